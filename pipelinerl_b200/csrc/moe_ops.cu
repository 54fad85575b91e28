// Routed feed-forward (mixture of experts) over a packed batch of n token rows, without a host round trip: the number
// of rows each expert gets stays on the device, so the whole layer can sit in a CUDA graph.
//
//   1. route:  (prl_moe_route, prl_moe_router) per row, the `top` experts with the largest router logits (ties: the lower
//              index), each with the weight sigmoid(logit) or softmax over the chosen; an optional bias per expert joins
//              the logits first; choice c of row t is the PAIR c * n + t.  prl_moe_choose (ready logits) and
//              prl_moe_router_choose instead rank the outputs by their softmax share or sigmoid plus a correction (which the
//              weights do not see), inside the best groups of outputs only; the weights may be divided by their sum;
//              outputs past the experts ("identity") hand the input through: their pairs are chosen and weighted like
//              the others but join no expert's rows.
//   2. group:  a stable counting sort of the pairs by expert (one CTA): perm[s] = pair at sorted place s, and a table
//              of row tiles (expert, first sorted place, rows <= 64) that the GEMMs walk; its length stays on the device.
//   3. grouped GEMM (twice):  C[row] = A[row'] * W_e^T for every tile, W_e = W + e * expert_stride.  The first product
//              reads the token's row (perm[s] % n) and writes sorted rows; the second reads sorted rows and writes
//              pair rows, i.e. `top` slices [top][n][width] that the sublayer's closing kernel adds up.
//      Batches with many rows per expert (bf16) gather the tokens' rows into sorted order first and run both products on
//      the tcgen05 CTA-pair kernel (prl_moe_gather, prl_moe_gemm_tc in gemm_tn.cu) with row tiles of 256.
//   4. gated activation of an expert with the pair's weight folded in: the weight multiplies the expert's INPUT, and
//              the two first projections are linear, so gate and up are scaled after the product (in fp32).
//
// Two GEMM kernels walk the same tile table.  fp32 operands (and sizes a 16-byte copy cannot express) take the
// CUDA-core kernel of gemm_any.cu with a row indirection: every output element is summed by one thread in ascending k.
// bf16 operands take a tensor-core kernel (mma.sync m16n8k16, fp32 accumulators): 64 x 128 output tile per CTA of eight
// warps, operands staged by cp.async (zero-filled past the edges) into a double buffer and read with ldmatrix.  A
// row's result depends only on the row and the expert's weights, never on which rows share its tile.
#include "prl_common.cuh"

namespace prl {
namespace {

constexpr int kTile = 64;
constexpr int kStepK = 16;

template <typename T> __device__ __forceinline__ float to_f32(T v);
template <> __device__ __forceinline__ float to_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f32<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }

__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }

// one warp per row; E up to 32 * kMaxPerLane
constexpr int kMaxPerLane = 32;
__global__ void moe_route_kernel(const float* __restrict__ logits, int64_t ld, const float* __restrict__ bias, int n, int E,
                                 int top, int softmax_weights, int32_t* __restrict__ sel, float* __restrict__ wsel) {
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x * (blockDim.x >> 5) + warp;
  if (t >= n) return;
  const float* z = logits + (int64_t)t * ld;
  uint32_t taken = 0;            // bit j: expert lane + 32 j already chosen
  float zsel_max = 0.f, denom = 0.f;
  for (int c = 0; c < top; ++c) {
    float best = -INFINITY;
    int arg = 0x7fffffff;
    for (int j = 0; j < kMaxPerLane; ++j) {
      const int e = lane + 32 * j;
      if (e >= E) break;
      if (taken >> j & 1u) continue;
      const float v = z[e] + (bias ? bias[e] : 0.f);
      if (v > best) { best = v; arg = e; }        // ascending e: the lower index wins a tie inside a lane
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ob = __shfl_xor_sync(0xffffffffu, best, o);
      const int oa = __shfl_xor_sync(0xffffffffu, arg, o);
      if (ob > best || (ob == best && oa < arg)) { best = ob; arg = oa; }
    }
    if ((arg & 31) == lane) taken |= 1u << (arg >> 5);
    if (c == 0) zsel_max = best;
    denom += expf(best - zsel_max);
    if (lane == 0) {
      sel[(int64_t)c * n + t] = arg;
      wsel[(int64_t)c * n + t] = softmax_weights ? expf(best - zsel_max) : sigmoid_f(best);
    }
  }
  if (softmax_weights == 2) {                    // softmax over ALL experts: the denominator sums every logit
    float all = 0.f;
    for (int j = 0; j < kMaxPerLane; ++j) {
      const int e = lane + 32 * j;
      if (e >= E) break;
      all += expf(z[e] + (bias ? bias[e] : 0.f) - zsel_max);
    }
    denom = warp_sum(all);
  }
  if (softmax_weights && lane == 0)
    for (int c = 0; c < top; ++c) wsel[(int64_t)c * n + t] /= denom;
}

// How a router's outputs are scored, ranked and weighted (prl_moe_choose, prl_moe_router_choose).
struct ChoiceRule {
  const float* correction;    // per output, joins the scores for the ranking only; NULL: none
  int top, groups, keep;      // `groups` equal groups of neighbours of which the `keep` best are open
  int group_top;              // a group is ranked by the sum of its `group_top` (1 or 2) best choice scores
  int sigmoid;                // score of an output: 1 the sigmoid of its logit, 0 its softmax share over all outputs
  int renorm;                 // 1: the chosen scores are divided by their sum (+ 1e-20)
  float scale;                // constant factor on the weights
};

// The choice for one row by one warp: c [E] and gs [groups] are the warp's scratch in shared memory, z [E] the logits.
// Outputs are ranked by score + correction, closed groups count as minus infinity; ties go to the lower index.
__device__ __forceinline__ void choose_row(const float* z, int E, const ChoiceRule& r, float* c, float* gs, int n, int t,
                                           int32_t* __restrict__ sel, float* __restrict__ wsel) {
  const int lane = threadIdx.x & 31;
  float zmax = 0.f, inv = 1.f;
  if (!r.sigmoid) {
    zmax = -INFINITY;
    for (int e = lane; e < E; e += 32) zmax = fmaxf(zmax, z[e]);
    zmax = warp_max(zmax);
    float sum = 0.f;
    for (int e = lane; e < E; e += 32) sum += expf(z[e] - zmax);
    inv = 1.f / warp_sum(sum);
  }
  auto score = [&](int e) { return r.sigmoid ? sigmoid_f(z[e]) : expf(z[e] - zmax) * inv; };
  for (int e = lane; e < E; e += 32) c[e] = score(e) + (r.correction ? r.correction[e] : 0.f);
  __syncwarp();
  auto best_of = [&](const float* v, int count) {          // index of the largest entry, the lowest on a tie
    float best = -INFINITY;
    int arg = 0x7fffffff;
    for (int e = lane; e < count; e += 32)
      if (v[e] > best) { best = v[e]; arg = e; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ob = __shfl_xor_sync(0xffffffffu, best, o);
      const int oa = __shfl_xor_sync(0xffffffffu, arg, o);
      if (ob > best || (ob == best && oa < arg)) { best = ob; arg = oa; }
    }
    return arg;
  };
  if (r.keep < r.groups) {
    const int size = E / r.groups;
    for (int g = lane; g < r.groups; g += 32) {
      float m = -INFINITY, m2 = -INFINITY;
      for (int e = 0; e < size; ++e) {
        const float v = c[g * size + e];
        m2 = fmaxf(m2, fminf(m, v));
        m = fmaxf(m, v);
      }
      gs[g] = (r.group_top > 1 && size > 1) ? m + m2 : m;
    }
    __syncwarp();
    for (int k = 0; k < r.keep; ++k) {                     // an open group is marked by taking it out of the ranking
      const int g = best_of(gs, r.groups);
      if (lane == 0 && g < r.groups) gs[g] = -INFINITY;
      __syncwarp();
    }
    for (int e = lane; e < E; e += 32)
      if (gs[e / size] != -INFINITY) c[e] = -INFINITY;     // still ranked: a closed group
    __syncwarp();
  }
  float total = 0.f, mine = 0.f;                           // lane k keeps choice k until the sum is known (up to 32 of them)
  for (int k = 0; k < r.top; ++k) {
    const int e = best_of(c, E);
    const bool ok = e < E;                                 // always, for finite logits
    const float w = ok ? score(e) : 0.f;
    total += w;
    if (lane == (k & 31)) {
      mine = w * r.scale;
      sel[(int64_t)k * n + t] = ok ? e : 0;
      if (r.top > 32) wsel[(int64_t)k * n + t] = mine;
      if (ok) c[e] = -INFINITY;
    }
    __syncwarp();
  }
  const float div = r.renorm ? total + 1e-20f : 1.f;
  if (r.top <= 32) {
    if (lane < r.top) wsel[(int64_t)lane * n + t] = mine / div;
  } else if (r.renorm) {
    for (int k = lane; k < r.top; k += 32) wsel[(int64_t)k * n + t] /= div;      // written by this lane
  }
}

// Choice from ready logits, one warp per row.
constexpr int kChooseWarps = 4;
__global__ void __launch_bounds__(kChooseWarps * 32) moe_choose_kernel(const float* __restrict__ logits, int64_t ld, int n, int E,
                                                                       ChoiceRule rule, int32_t* __restrict__ sel,
                                                                       float* __restrict__ wsel) {
  pdl_wait();
  extern __shared__ float csm[];                 // per warp: [E] choice scores | [groups] group scores
  const int warp = threadIdx.x >> 5;
  const int t = blockIdx.x * kChooseWarps + warp;
  if (t >= n) return;
  float* c = csm + (size_t)warp * (E + rule.groups);
  choose_row(logits + (int64_t)t * ld, E, rule, c, c + E, n, t, sel, wsel);
}

// Router and choice in one kernel: logits[e] = x . Wr[e] in fp32 (block per row, warps
// take experts in turn, a lane sums every 32nd group of channels, then the warp's shuffle tree: a fixed order), then the top-k
// pass of moe_route_kernel over the logits in shared memory (RULED: choose_row instead, with scratch behind the logits).
template <typename TX, typename TW, bool RULED>
__global__ void __launch_bounds__(256) moe_router_kernel(const TX* __restrict__ x, const TW* __restrict__ Wr,
                                                         const float* __restrict__ bias, int n, int W, int E, int top,
                                                         int softmax_weights, ChoiceRule rule, int32_t* __restrict__ sel,
                                                         float* __restrict__ wsel) {
  pdl_wait();
  extern __shared__ __align__(16) float rsm[];       // [W] the row | [E] logits | RULED: [E] choice scores | [groups] group scores
  float* xs = rsm;
  float* z = rsm + W;
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  constexpr int V = 16 / sizeof(TW);              // router weights per 16-byte load
  const bool vec = W % V == 0 && ((uintptr_t)Wr & 15) == 0;
  // one element type and aligned rows: the row is read beside the weights (from L1 for all warps but the first), not staged
  const bool direct = sizeof(TX) == sizeof(TW) && vec && ((uintptr_t)x & 15) == 0;
  if (!direct) {
    for (int c = threadIdx.x; c < W; c += blockDim.x) xs[c] = to_f32(x[(int64_t)t * W + c]);
    __syncthreads();
  }
  for (int e = warp; e < E; e += nw) {
    const TW* w = Wr + (int64_t)e * W;
    float a = 0.f;
    if (direct) {                                 // a lane sums its channels in ascending order
      const TX* xr = x + (int64_t)t * W;
#pragma unroll 4
      for (int c = V * lane; c < W; c += 32 * V) {
        const uint4 raw = *reinterpret_cast<const uint4*>(w + c), xraw = *reinterpret_cast<const uint4*>(xr + c);
        const TW* wv = reinterpret_cast<const TW*>(&raw);
        const TX* xv = reinterpret_cast<const TX*>(&xraw);
#pragma unroll
        for (int j = 0; j < V; ++j) a = fmaf(to_f32(xv[j]), to_f32(wv[j]), a);
      }
    } else if (vec) {
#pragma unroll 4
      for (int c = V * lane; c < W; c += 32 * V) {
        const uint4 raw = *reinterpret_cast<const uint4*>(w + c);
        const TW* wv = reinterpret_cast<const TW*>(&raw);
#pragma unroll
        for (int j = 0; j < V; j += 4) {
          const float4 xv = *reinterpret_cast<const float4*>(xs + c + j);
          a = fmaf(xv.x, to_f32(wv[j]), a); a = fmaf(xv.y, to_f32(wv[j + 1]), a);
          a = fmaf(xv.z, to_f32(wv[j + 2]), a); a = fmaf(xv.w, to_f32(wv[j + 3]), a);
        }
      }
    } else {
#pragma unroll 8
      for (int c = lane; c < W; c += 32) a = fmaf(xs[c], to_f32(w[c]), a);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) a += __shfl_xor_sync(0xffffffffu, a, o);
    if (lane == 0) z[e] = a + (bias ? bias[e] : 0.f);
  }
  __syncthreads();
  if (warp != 0) return;
  if constexpr (RULED) {
    choose_row(z, E, rule, z + E, z + 2 * E, n, t, sel, wsel);
    return;
  }
  uint32_t taken = 0;
  float zsel_max = 0.f, denom = 0.f;
  for (int c = 0; c < top; ++c) {
    float best = -INFINITY;
    int arg = 0x7fffffff;
    for (int j = 0; j < kMaxPerLane; ++j) {
      const int e = lane + 32 * j;
      if (e >= E) break;
      if (taken >> j & 1u) continue;
      const float v = z[e];
      if (v > best) { best = v; arg = e; }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ob = __shfl_xor_sync(0xffffffffu, best, o);
      const int oa = __shfl_xor_sync(0xffffffffu, arg, o);
      if (ob > best || (ob == best && oa < arg)) { best = ob; arg = oa; }
    }
    if ((arg & 31) == lane) taken |= 1u << (arg >> 5);
    if (c == 0) zsel_max = best;
    denom += expf(best - zsel_max);
    if (lane == 0) {
      sel[(int64_t)c * n + t] = arg;
      wsel[(int64_t)c * n + t] = softmax_weights ? expf(best - zsel_max) : sigmoid_f(best);
    }
  }
  if (softmax_weights == 2) {                    // softmax over ALL experts: the denominator sums every logit
    float all = 0.f;
    for (int j = 0; j < kMaxPerLane; ++j) {
      const int e = lane + 32 * j;
      if (e >= E) break;
      all += expf(z[e] - zsel_max);
    }
    denom = warp_sum(all);
  }
  if (softmax_weights && lane == 0)
    for (int c = 0; c < top; ++c) wsel[(int64_t)c * n + t] /= denom;
}

// meta[0] = number of tiles, meta[1] = sorted pairs; tiles[3 * i + {0, 1, 2}] = expert, first sorted place, rows (<= tile_rows)
__global__ void __launch_bounds__(1024) moe_group_kernel(const int32_t* __restrict__ sel, int pairs, int E, int tile_rows,
                                                         int32_t* __restrict__ perm, int32_t* __restrict__ meta,
                                                         int32_t* __restrict__ tiles) {
  pdl_wait();
  extern __shared__ int32_t cnt[];      // [E] counts, then [E] offsets
  int32_t* off = cnt + E;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, nw = blockDim.x >> 5;
  for (int e = tid; e < E; e += blockDim.x) cnt[e] = 0;
  __syncthreads();
  for (int p = tid; p < pairs; p += blockDim.x)
    if (sel[p] < E) atomicAdd(&cnt[sel[p]], 1);          // a choice past the experts belongs to none of them
  __syncthreads();
  if (tid == 0) {
    int at = 0, nt = 0;
    for (int e = 0; e < E; ++e) {
      off[e] = at;
      for (int r0 = 0; r0 < cnt[e]; r0 += tile_rows) {
        tiles[3 * nt] = e;
        tiles[3 * nt + 1] = at + r0;
        tiles[3 * nt + 2] = min(tile_rows, cnt[e] - r0);
        ++nt;
      }
      at += cnt[e];
    }
    meta[0] = nt;
    meta[1] = at;
  }
  __syncthreads();
  for (int e = warp; e < E; e += nw) {     // stable: pairs of an expert keep their order
    int at = off[e];
    for (int p0 = 0; p0 < pairs; p0 += 32) {
      const int p = p0 + lane;
      const bool mine = p < pairs && sel[p] == e;
      const uint32_t mask = __ballot_sync(0xffffffffu, mine);
      if (mine) perm[at + __popc(mask & ((1u << lane) - 1u))] = p;
      at += __popc(mask);
    }
  }
}

// The same for up to kGroupExperts experts: every warp counts a run of the pairs, then places them behind the runs of the warps
// before it (a warp finds its lanes of one expert with a match, so the order stays that of the pairs).
constexpr int kGroupExperts = 256, kGroupWarps = 32;
__global__ void __launch_bounds__(32 * kGroupWarps) moe_group_runs_kernel(const int32_t* __restrict__ sel, int pairs, int E, int tile_rows,
                                                                         int32_t* __restrict__ perm, int32_t* __restrict__ meta,
                                                                         int32_t* __restrict__ tiles) {
  pdl_wait();
  extern __shared__ int32_t cnt[];      // [warps][E] counts, then first places; [E] totals; [E] first place and first tile
  int32_t* total = cnt + kGroupWarps * E;
  int32_t* off = total + E;
  int32_t* tile0 = off + E;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  int32_t* mine = cnt + warp * E;
  for (int i = tid; i < kGroupWarps * E; i += blockDim.x) cnt[i] = 0;
  __syncthreads();
  const int run = (pairs + 32 * kGroupWarps - 1) / (32 * kGroupWarps) * 32, p_end = min(pairs, (warp + 1) * run);
  for (int p0 = warp * run; p0 < p_end; p0 += 32) {
    const int p = p0 + lane, e = p < p_end ? sel[p] : 0x7fffffff;
    const uint32_t same = __match_any_sync(0xffffffffu, e);
    if (e < E && lane == __ffs(same) - 1) mine[e] += __popc(same);       // a choice past the experts belongs to none of them
    __syncwarp();
  }
  __syncthreads();
  for (int e = tid; e < E; e += blockDim.x) {
    int at = 0;
    for (int w = 0; w < kGroupWarps; ++w) {
      const int c = cnt[w * E + e];
      cnt[w * E + e] = at;
      at += c;
    }
    total[e] = at;
  }
  __syncthreads();
  if (warp == 0) {                      // first place and first tile of every expert: running sums, 32 experts at a time
    int at = 0, nt = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
      const int c = e0 + lane < E ? total[e0 + lane] : 0, k = (c + tile_rows - 1) / tile_rows;
      int sc = c, sk = k;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int vc = __shfl_up_sync(0xffffffffu, sc, o), vk = __shfl_up_sync(0xffffffffu, sk, o);
        if (lane >= o) { sc += vc; sk += vk; }
      }
      if (e0 + lane < E) { off[e0 + lane] = at + sc - c; tile0[e0 + lane] = nt + sk - k; }
      at += __shfl_sync(0xffffffffu, sc, 31);
      nt += __shfl_sync(0xffffffffu, sk, 31);
    }
    if (lane == 0) { meta[0] = nt; meta[1] = at; }
  }
  __syncthreads();
  for (int e = tid; e < E; e += blockDim.x)
    for (int r0 = 0, i = tile0[e]; r0 < total[e]; r0 += tile_rows, ++i) {
      tiles[3 * i] = e;
      tiles[3 * i + 1] = off[e] + r0;
      tiles[3 * i + 2] = min(tile_rows, total[e] - r0);
    }
  for (int p0 = warp * run; p0 < p_end; p0 += 32) {
    const int p = p0 + lane, e = p < p_end ? sel[p] : 0x7fffffff;
    const uint32_t same = __match_any_sync(0xffffffffu, e);
    const int first = e < E ? mine[e] : 0;
    __syncwarp();
    if (e < E) {
      perm[off[e] + first + __popc(same & ((1u << lane) - 1u))] = p;
      if (lane == __ffs(same) - 1) mine[e] = first + __popc(same);
    }
    __syncwarp();
  }
}

// out[s] = x[perm[s] % n]: the tokens' rows (16-byte units) in sorted order, the A operand of the tcgen05 grouped GEMM
__global__ void __launch_bounds__(128) moe_gather_kernel(const uint4* __restrict__ x, const int32_t* __restrict__ perm,
                                                         const int32_t* __restrict__ meta, int n, int units, uint4* __restrict__ out) {
  pdl_wait();
  const int s = blockIdx.x;
  if (s >= meta[1]) return;
  const uint4* src = x + (int64_t)(perm[s] % n) * units;
  uint4* dst = out + (int64_t)s * units;
#pragma unroll 4
  for (int i = threadIdx.x; i < units; i += 128) dst[i] = src[i];
}

// ACT: what the product becomes before it is stored.  kActNone: C fp32, the product itself; otherwise C is the next
// product's operand (type TA), C[row] = act(product) * wsel[pair]
constexpr int kActNone = 0, kActRelu2 = 1, kActGelu = 2;      // relu(z)^2 | z Phi(z), the error-function form
template <int ACT> __device__ __forceinline__ float expert_act(float z) {
  if constexpr (ACT == kActRelu2) {
    const float r = fmaxf(z, 0.f);
    return r * r;
  } else {
    return 0.5f * z * (1.f + erff(z * 0.70710678118654752f));
  }
}

template <typename TA, typename TW, int ACT>
__global__ void __launch_bounds__(256) moe_gemm_kernel(const TA* __restrict__ A, int64_t lda, int a_mod,
                                                       const TW* __restrict__ W, int64_t expert_stride, int64_t ldw,
                                                       const int32_t* __restrict__ perm, const int32_t* __restrict__ meta,
                                                       const int32_t* __restrict__ tiles, int N, int K,
                                                       void* __restrict__ C_v, int64_t ldc, int c_perm,
                                                       const float* __restrict__ wsel) {
  pdl_wait();
  const int tile = blockIdx.y;
  if (tile >= meta[0]) return;
  __shared__ float As[kStepK][kTile + 4];
  __shared__ float Ws[kStepK][kTile + 4];
  __shared__ int32_t a_row[kTile], c_row[kTile];
  __shared__ float c_w[kTile];
  const int e = tiles[3 * tile], s0 = tiles[3 * tile + 1], M = tiles[3 * tile + 2];
  const int tid = threadIdx.x;
  if (tid < kTile) {
    const int s = s0 + min(tid, M - 1);
    const int p = perm[s];
    if constexpr (ACT != kActNone) c_w[tid] = wsel[p];
    a_row[tid] = a_mod > 0 ? p % a_mod : s;
    c_row[tid] = c_perm ? p : s;
  }
  __syncthreads();
  const TW* We = W + (int64_t)e * expert_stride;
  const int n0 = blockIdx.x * kTile;
  const int tm = (tid / 16) * 4, tn = (tid % 16) * 4;
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  const int lr = tid / 4;          // 0..63
  const int lk = (tid % 4) * 4;    // 0,4,8,12
  const int64_t arow = a_row[lr];
  for (int k0 = 0; k0 < K; k0 += kStepK) {
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int k = k0 + lk + j;
      const int nn = n0 + lr;
      As[lk + j][lr] = (lr < M && k < K) ? to_f32(A[arow * lda + k]) : 0.f;
      Ws[lk + j][lr] = (nn < N && k < K) ? to_f32(We[(int64_t)nn * ldw + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < kStepK; ++kk) {
      float a[4], w[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) a[i] = As[kk][tm + i];
#pragma unroll
      for (int j = 0; j < 4; ++j) w[j] = Ws[kk][tn + j];
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], w[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    if (tm + i >= M) continue;
    const int64_t row = c_row[tm + i];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int nn = n0 + tn + j;
      if (nn >= N) continue;
      if constexpr (ACT != kActNone) {
        reinterpret_cast<TA*>(C_v)[row * ldc + nn] = TA(expert_act<ACT>(acc[i][j]) * c_w[tm + i]);
      } else {
        reinterpret_cast<float*>(C_v)[row * ldc + nn] = acc[i][j];
      }
    }
  }
}

// ---- bf16 tensor-core variant ------------------------------------------------------------------------------------------
constexpr int kBN = 128, kBK = 64, kPad = 8;      // tile N, K step, padding (halves) that keeps ldmatrix conflict-free
constexpr int kLds = kBK + kPad;                  // 72 halves = 144 bytes per staged row
constexpr int kStages = 4;                        // cp.async stages in flight: a few-row tile is a pure weight stream
constexpr size_t kMmaSmem = (size_t)kStages * (kTile + kBN) * kLds * sizeof(__nv_bfloat16);

__device__ __forceinline__ void cp_async16_zfill(void* dst, const void* src, int bytes) {
  const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void ldsm_x4(uint32_t (&r)[4], const void* p) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

template <int ACT>
__global__ void __launch_bounds__(256) moe_gemm_mma_kernel(const __nv_bfloat16* __restrict__ A, int64_t lda, int a_mod,
                                                           const __nv_bfloat16* __restrict__ W, int64_t expert_stride,
                                                           int64_t ldw, const int32_t* __restrict__ perm,
                                                           const int32_t* __restrict__ meta, const int32_t* __restrict__ tiles,
                                                           int N, int K, void* __restrict__ C_v, int64_t ldc, int c_perm,
                                                           const float* __restrict__ wsel) {
  pdl_wait();
  const int tile = blockIdx.y;
  if (tile >= meta[0]) return;
  extern __shared__ __align__(16) unsigned char mma_smem[];
  typedef __nv_bfloat16 (*ATile)[kTile][kLds];
  typedef __nv_bfloat16 (*BTile)[kBN][kLds];
  ATile As = reinterpret_cast<ATile>(mma_smem);                                           // [kStages][64][72]
  BTile Bs = reinterpret_cast<BTile>(mma_smem + (size_t)kStages * kTile * kLds * sizeof(__nv_bfloat16));   // [kStages][128][72]
  __shared__ int32_t a_row[kTile], c_row[kTile];
  __shared__ float c_w[kTile];
  const int e = tiles[3 * tile], s0 = tiles[3 * tile + 1], M = tiles[3 * tile + 2];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  if (tid < kTile) {
    const int s = s0 + min(tid, M - 1);
    const int p = perm[s];
    if constexpr (ACT != kActNone) c_w[tid] = wsel[p];
    a_row[tid] = a_mod > 0 ? p % a_mod : s;
    c_row[tid] = c_perm ? p : s;
  }
  __syncthreads();
  const __nv_bfloat16* We = W + (int64_t)e * expert_stride;
  const int n0 = blockIdx.x * kBN;
  const int wm = (warp >> 2) * 32, wn = (warp & 3) * 32;       // warp tile 32 x 32
  float acc[2][4][4];
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int q = 0; q < 4; ++q) acc[i][j][q] = 0.f;
  // loaders: A 64 rows x 8 chunks of 8 halves (two per thread), B 128 rows x 8 chunks (four per thread)
  const int lr = tid >> 3, lc = (tid & 7) * 8;
  const int64_t a_off[2] = {(int64_t)a_row[lr] * lda, (int64_t)a_row[lr + 32] * lda};
  auto stage = [&](int k0, int buf) {
    const int k = k0 + lc;
    const bool kin = k < K;
#pragma unroll
    for (int h = 0; h < 2; ++h)
      if (32 * h < M)         // uniform: the upper half of a short tile is not staged, and the warps that own it do nothing
        cp_async16_zfill(&As[buf][lr + 32 * h][lc], A + a_off[h] + (kin ? k : 0), (kin && lr + 32 * h < M) ? 16 : 0);
#pragma unroll
    for (int h = 0; h < 4; ++h) {
      const int r = lr + 32 * h, nn = n0 + r;
      const bool ok = kin && nn < N;
      cp_async16_zfill(&Bs[buf][r][lc], We + (int64_t)(ok ? nn : 0) * ldw + (kin ? k : 0), ok ? 16 : 0);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  // kStages - 1 steps in flight; a commit per step keeps the group count regular (empty past the end, where `stage`
  // copies nothing but zero fill into a buffer nobody reads)
#pragma unroll
  for (int st = 0; st < kStages - 1; ++st) stage(st * kBK, st);
  int buf = 0;
  for (int k0 = 0; k0 < K; k0 += kBK, buf = (buf + 1) % kStages) {
    asm volatile("cp.async.wait_group %0;" ::"n"(kStages - 2) : "memory");
    __syncthreads();            // step k0 has landed for every thread, and every warp is done with the buffer refilled next
    stage(k0 + (kStages - 1) * kBK, (buf + kStages - 1) % kStages);
    if (wm < M)                 // warp-uniform
#pragma unroll
    for (int kk = 0; kk < kBK; kk += 16) {
      uint32_t af[2][4], bf[2][4];
#pragma unroll
      for (int i = 0; i < 2; ++i) ldsm_x4(af[i], &As[buf][wm + 16 * i + (lane & 15)][kk + (lane >> 4) * 8]);
#pragma unroll
      for (int j = 0; j < 2; ++j) ldsm_x4(bf[j], &Bs[buf][wn + 16 * j + (lane & 7) + ((lane >> 4) << 3)][kk + ((lane >> 3) & 1) * 8]);
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) mma_bf16(acc[i][j], af[i], bf[j >> 1][(j & 1) * 2], bf[j >> 1][(j & 1) * 2 + 1]);
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int m = wm + 16 * i + (lane >> 2) + 8 * half;
      if (m >= M) continue;
      const int64_t at = (int64_t)c_row[m] * ldc;
      if constexpr (ACT != kActNone) {
        __nv_bfloat16* crow = reinterpret_cast<__nv_bfloat16*>(C_v) + at;
        const float w = c_w[m];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int nn = n0 + wn + 8 * j + (lane & 3) * 2;
          if (nn < N) crow[nn] = __float2bfloat16_rn(expert_act<ACT>(acc[i][j][2 * half]) * w);
          if (nn + 1 < N) crow[nn + 1] = __float2bfloat16_rn(expert_act<ACT>(acc[i][j][2 * half + 1]) * w);
        }
        continue;
      }
      float* crow = reinterpret_cast<float*>(C_v) + at;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int nn = n0 + wn + 8 * j + (lane & 3) * 2;
        if (nn < N) crow[nn] = acc[i][j][2 * half];
        if (nn + 1 < N) crow[nn + 1] = acc[i][j][2 * half + 1];
      }
    }
}

// act[s] = g * sigmoid(beta g) * (u + 1),  g = min(w * gate, lim), u = clamp(w * up, -lim, lim),  w = wsel[perm[s]]
template <typename T>
__global__ void moe_glu_kernel(const float* __restrict__ gu, int64_t ld, int F, const int32_t* __restrict__ perm,
                               const float* __restrict__ wsel, float lim, float beta, T* __restrict__ out) {
  pdl_wait();
  const int64_t s = blockIdx.x;
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= F) return;
  const float w = wsel[perm[s]];
  const float g = fminf(w * gu[s * ld + c], lim);
  const float u = fminf(fmaxf(w * gu[s * ld + F + c], -lim), lim);
  out[s * F + c] = T(g * sigmoid_f(beta * g) * (u + 1.f));
}

// act[s] = act(gate) * up * (w * wscale), act = SiLU: the pair's weight multiplies the expert's OUTPUT; the second
// projection is linear and has no bias, so the weight is applied to its input instead (in fp32, before the rounding)
template <typename T>
__global__ void moe_glu_out_kernel(const float* __restrict__ gu, int64_t ld, int F, const int32_t* __restrict__ perm,
                                   const float* __restrict__ wsel, float wscale, T* __restrict__ out) {
  pdl_wait();
  const int64_t s = blockIdx.x;
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= F) return;
  const float w = wsel[perm[s]] * wscale;
  const float g = gu[s * ld + c];
  out[s * F + c] = T(g * sigmoid_f(g) * gu[s * ld + F + c] * w);
}

}  // namespace
}  // namespace prl

using namespace prl;
typedef __nv_bfloat16 bf16;

static cudaError_t launch_group(const int32_t* sel, int pairs, int experts, int tile_rows, int32_t* perm, int32_t* meta, int32_t* tiles,
                                cudaStream_t s) {
  if (experts <= kGroupExperts)
    return launch_pdl(moe_group_runs_kernel, dim3(1), dim3(32 * kGroupWarps), (size_t)(kGroupWarps + 3) * experts * sizeof(int32_t), s, sel,
                      pairs, experts, tile_rows, perm, meta, tiles);
  return launch_pdl(moe_group_kernel, dim3(1), dim3(1024), (size_t)(2 * experts * sizeof(int32_t)), s, sel, pairs, experts, tile_rows, perm,
                    meta, tiles);
}

extern "C" int64_t prl_moe_max_tiles(int64_t pairs, int32_t experts) { return (pairs + kTile - 1) / kTile + experts; }

extern "C" int prl_moe_route(const float* logits, int64_t ld, const float* bias, int32_t n, int32_t experts, int32_t top,
                             int32_t softmax_weights, int32_t* sel, float* wsel, int32_t* perm, int32_t* meta,
                             int32_t* tiles, prl_stream_t st) {
  PRL_CHECK_ARG(logits && sel && wsel && perm && meta && tiles, "prl_moe_route: NULL argument");
  PRL_CHECK_ARG(n >= 1 && experts >= 1 && experts <= 32 * kMaxPerLane && top >= 1 && top <= experts && ld >= experts,
                "prl_moe_route: bad shape (experts=%d top=%d; at most %d experts)", experts, top, 32 * kMaxPerLane);
  cudaStream_t s = (cudaStream_t)st;
  PRL_CUDA(launch_pdl(moe_route_kernel, dim3((n + 7) / 8), dim3(256), (size_t)0, s, logits, ld, bias, n, experts, top, softmax_weights, sel, wsel));
  PRL_LAUNCH_CHECK();
  PRL_CUDA(launch_group(sel, n * top, experts, kTile, perm, meta, tiles, s));
  PRL_LAUNCH_CHECK();
  return PRL_OK;
}

// Router product, choice and grouping in two launches: x [n, W] and the router matrix [experts, W] in fp32 or bf16.
// Needs (W + experts) * 4 bytes of shared memory; returns PRL_ERR_INVALID beyond 160 KB (use prl_gemm_any + prl_moe_route).
static int moe_router_impl(const void* x, int32_t x_is_f32, const void* Wr, int32_t w_is_f32, const float* bias, int32_t n, int32_t W,
                           int32_t experts, int32_t outputs, int32_t top, int32_t softmax_weights, const ChoiceRule* rule,
                           int32_t tile_rows, int32_t* sel, float* wsel, int32_t* perm, int32_t* meta, int32_t* tiles, prl_stream_t st) {
  PRL_CHECK_ARG(x && Wr && sel && wsel && perm && meta && tiles, "prl_moe_router: NULL argument");
  PRL_CHECK_ARG(n >= 1 && W >= 1 && outputs >= 1 && outputs <= 32 * kMaxPerLane && top >= 1 && top <= outputs,
                "prl_moe_router: bad shape (outputs=%d top=%d; at most %d outputs)", outputs, top, 32 * kMaxPerLane);
  const size_t smem = ((size_t)W + outputs + (rule ? outputs + rule->groups : 0)) * sizeof(float);
  PRL_CHECK_ARG(smem <= 160 * 1024, "prl_moe_router: a row of %d channels does not fit in shared memory", W);
  cudaStream_t s = (cudaStream_t)st;
  static SmemAttr attr[8] = {};
#define PRL_RT(TX, TW, RULED, I)                                                                                       \
  do {                                                                                                                 \
    if (smem > 48 * 1024) PRL_CUDA(ensure_smem(moe_router_kernel<TX, TW, RULED>, (int)smem, attr[I]));                 \
    PRL_CUDA(launch_pdl((moe_router_kernel<TX, TW, RULED>), dim3(n), dim3(256), smem, s, (const TX*)x, (const TW*)Wr, bias, n, W, \
                        outputs, top, softmax_weights, rule ? *rule : ChoiceRule{}, sel, wsel));                       \
  } while (0)
#define PRL_RT2(TX, TW, I)                \
  do {                                    \
    if (rule) PRL_RT(TX, TW, true, I);    \
    else PRL_RT(TX, TW, false, I + 4);    \
  } while (0)
  if (x_is_f32 && w_is_f32) PRL_RT2(float, float, 0);
  else if (x_is_f32) PRL_RT2(float, bf16, 1);
  else if (w_is_f32) PRL_RT2(bf16, float, 2);
  else PRL_RT2(bf16, bf16, 3);
#undef PRL_RT2
#undef PRL_RT
  PRL_LAUNCH_CHECK();
  PRL_CUDA(launch_group(sel, n * top, experts, tile_rows, perm, meta, tiles, s));
  PRL_LAUNCH_CHECK();
  return PRL_OK;
}

extern "C" int prl_moe_router(const void* x, int32_t x_is_f32, const void* Wr, int32_t w_is_f32, const float* bias, int32_t n, int32_t W,
                              int32_t experts, int32_t top, int32_t softmax_weights, int32_t* sel, float* wsel, int32_t* perm,
                              int32_t* meta, int32_t* tiles, prl_stream_t st) {
  return moe_router_impl(x, x_is_f32, Wr, w_is_f32, bias, n, W, experts, experts, top, softmax_weights, nullptr, kTile, sel, wsel, perm,
                         meta, tiles, st);
}

static bool choice_rule_ok(int experts, int outputs, const ChoiceRule& r) {
  return experts >= 1 && outputs >= experts && outputs <= 1024 && r.groups >= 1 && outputs % r.groups == 0 && r.keep >= 1 &&
         r.keep <= r.groups && r.top >= 1 && r.top <= outputs / r.groups * r.keep && (r.group_top == 1 || r.group_top == 2);
}

// prl_moe_router with the scoring, ranking and weighting of prl_moe_choose (router rows = outputs).
extern "C" int prl_moe_router_choose(const void* x, int32_t x_is_f32, const void* Wr, int32_t w_is_f32, const float* correction, int32_t n,
                                     int32_t W, int32_t experts, int32_t outputs, int32_t top, int32_t groups, int32_t keep,
                                     int32_t group_top, int32_t sigmoid, int32_t renorm, float scale, int32_t tile_rows, int32_t* sel,
                                     float* wsel, int32_t* perm, int32_t* meta, int32_t* tiles, prl_stream_t st) {
  const ChoiceRule rule{correction, top, groups, keep, group_top, sigmoid, renorm, scale};
  PRL_CHECK_ARG(choice_rule_ok(experts, outputs, rule) && (tile_rows == kTile || tile_rows == 256),
                "prl_moe_router_choose: bad shape (experts=%d outputs=%d top=%d groups=%d keep=%d)", experts, outputs, top, groups, keep);
  return moe_router_impl(x, x_is_f32, Wr, w_is_f32, nullptr, n, W, experts, outputs, top, 0, &rule, tile_rows, sel, wsel, perm, meta,
                         tiles, st);
}

// Choice among outputs whose logits are already there (columns of a projection buffer), and the grouping of the pairs by expert:
// `outputs` = experts + identity outputs; see ChoiceRule.  tile_rows: 64 for prl_moe_gemm, 256 for prl_moe_gemm_tc.  keep == groups (e.g. 1, 1): every output is open.
extern "C" int prl_moe_choose(const float* logits, int64_t ld, const float* correction, int32_t n, int32_t experts, int32_t outputs,
                              int32_t top, int32_t groups, int32_t keep, int32_t group_top, int32_t sigmoid, int32_t renorm, float scale,
                              int32_t tile_rows, int32_t* sel, float* wsel, int32_t* perm, int32_t* meta, int32_t* tiles,
                              prl_stream_t st) {
  PRL_CHECK_ARG(tile_rows == kTile || tile_rows == 256, "prl_moe_choose: row tiles of 64 or 256");
  PRL_CHECK_ARG(logits && sel && wsel && perm && meta && tiles, "prl_moe_choose: NULL argument");
  const ChoiceRule rule{correction, top, groups, keep, group_top, sigmoid, renorm, scale};
  PRL_CHECK_ARG(n >= 1 && ld >= outputs && choice_rule_ok(experts, outputs, rule),
                "prl_moe_choose: bad shape (experts=%d outputs=%d top=%d groups=%d keep=%d)", experts, outputs, top, groups, keep);
  cudaStream_t s = (cudaStream_t)st;
  PRL_CUDA(launch_pdl(moe_choose_kernel, dim3((n + kChooseWarps - 1) / kChooseWarps), dim3(kChooseWarps * 32),
                      (size_t)kChooseWarps * (outputs + groups) * sizeof(float), s, logits, ld, n, outputs, rule, sel, wsel));
  PRL_LAUNCH_CHECK();
  PRL_CUDA(launch_group(sel, n * top, experts, tile_rows, perm, meta, tiles, s));
  PRL_LAUNCH_CHECK();
  return PRL_OK;
}

extern "C" int prl_moe_gather(const void* x_bf16, const int32_t* perm, const int32_t* meta, int32_t n, int32_t pairs, int32_t W, void* out,
                              prl_stream_t st) {
  PRL_CHECK_ARG(x_bf16 && perm && meta && out && n >= 1 && pairs >= 1 && W >= 8 && W % 8 == 0 && (((uintptr_t)x_bf16 | (uintptr_t)out) & 15) == 0,
                "prl_moe_gather: bad argument (rows of a multiple of eight bf16)");
  PRL_CUDA(launch_pdl(moe_gather_kernel, dim3(pairs), dim3(128), (size_t)0, (cudaStream_t)st, (const uint4*)x_bf16, perm, meta, n, W / 8, (uint4*)out));
  PRL_LAUNCH_CHECK();
  return PRL_OK;
}

template <int ACT>
static int moe_gemm_impl(const void* A, int32_t a_is_f32, int64_t lda, int32_t a_mod, const void* W, int32_t w_is_f32,
                         int64_t expert_stride, int64_t ldw, const int32_t* perm, const int32_t* meta, const int32_t* tiles,
                         int64_t max_tiles, int64_t N, int64_t K, void* C, int64_t ldc, int32_t c_perm, const float* wsel,
                         prl_stream_t st) {
  PRL_CHECK_ARG(A && W && perm && meta && tiles && C && (ACT == kActNone || wsel), "prl_moe_gemm: NULL argument");
  PRL_CHECK_ARG(max_tiles >= 1 && max_tiles <= 65535 && N >= 1 && K >= 1 && lda >= K && ldw >= K && ldc >= N && a_mod >= 0,
                "prl_moe_gemm: bad shape (tiles=%lld N=%lld K=%lld)", (long long)max_tiles, (long long)N, (long long)K);
  cudaStream_t s = (cudaStream_t)st;
  if (!a_is_f32 && !w_is_f32 && K % 8 == 0 && lda % 8 == 0 && ldw % 8 == 0 && expert_stride % 8 == 0 &&
      ((uintptr_t)A & 15) == 0 && ((uintptr_t)W & 15) == 0) {
    dim3 grid_tc((unsigned)((N + kBN - 1) / kBN), (unsigned)max_tiles);
    static SmemAttr attr = {};
    PRL_CUDA(ensure_smem(moe_gemm_mma_kernel<ACT>, (int)kMmaSmem, attr));
    PRL_CUDA(launch_pdl(moe_gemm_mma_kernel<ACT>, grid_tc, dim3(256), kMmaSmem, s, (const bf16*)A, lda, a_mod, (const bf16*)W,
                        expert_stride, ldw, perm, meta, tiles, (int)N, (int)K, C, ldc, c_perm, wsel));
    PRL_LAUNCH_CHECK();
    return PRL_OK;
  }
  dim3 grid((unsigned)((N + kTile - 1) / kTile), (unsigned)max_tiles);
#define PRL_MG(TA, TW) PRL_CUDA(launch_pdl((moe_gemm_kernel<TA, TW, ACT>), grid, dim3(256), (size_t)0, s, (const TA*)A, lda, a_mod, (const TW*)W, \
                                           expert_stride, ldw, perm, meta, tiles, (int)N, (int)K, C, ldc, c_perm, wsel))
  if (a_is_f32 && w_is_f32) PRL_MG(float, float);
  else if (a_is_f32) PRL_MG(float, bf16);
  else if (w_is_f32) PRL_MG(bf16, float);
  else PRL_MG(bf16, bf16);
#undef PRL_MG
  PRL_LAUNCH_CHECK();
  return PRL_OK;
}

extern "C" int prl_moe_gemm(const void* A, int32_t a_is_f32, int64_t lda, int32_t a_mod, const void* W, int32_t w_is_f32,
                            int64_t expert_stride, int64_t ldw, const int32_t* perm, const int32_t* meta,
                            const int32_t* tiles, int64_t max_tiles, int64_t N, int64_t K, float* C, int64_t ldc,
                            int32_t c_perm, prl_stream_t st) {
  return moe_gemm_impl<kActNone>(A, a_is_f32, lda, a_mod, W, w_is_f32, expert_stride, ldw, perm, meta, tiles, max_tiles, N, K, C, ldc,
                              c_perm, nullptr, st);
}

// First product of ungated experts: out[s] = act(A[row of s] W_e^T) * wsel[pair of s], in the operand type of A and in sorted
// order, i.e. the second product's operand (its weight on the expert's OUTPUT: that product is linear).  act 1: relu(z)^2,
// 2: gelu(z) in its error-function form.
extern "C" int prl_moe_gemm_act(const void* A, int32_t a_is_f32, int64_t lda, int32_t a_mod, const void* W, int32_t w_is_f32,
                                int64_t expert_stride, int64_t ldw, const int32_t* perm, const int32_t* meta,
                                const int32_t* tiles, int64_t max_tiles, int64_t N, int64_t K, int32_t act, const float* wsel,
                                void* out, int64_t ld_out, prl_stream_t st) {
  PRL_CHECK_ARG(act == kActRelu2 || act == kActGelu, "prl_moe_gemm_act: unknown activation %d", act);
  return act == kActRelu2 ? moe_gemm_impl<kActRelu2>(A, a_is_f32, lda, a_mod, W, w_is_f32, expert_stride, ldw, perm, meta, tiles, max_tiles,
                                                     N, K, out, ld_out, 0, wsel, st)
                          : moe_gemm_impl<kActGelu>(A, a_is_f32, lda, a_mod, W, w_is_f32, expert_stride, ldw, perm, meta, tiles, max_tiles,
                                                    N, K, out, ld_out, 0, wsel, st);
}

extern "C" int prl_moe_glu(const float* gate_up, int64_t ld, int64_t pairs, int32_t F, const int32_t* perm,
                           const float* wsel, float limit, float beta, void* out, int32_t f32, prl_stream_t st) {
  PRL_CHECK_ARG(gate_up && perm && wsel && out && pairs >= 1 && F >= 1 && ld >= 2 * (int64_t)F, "prl_moe_glu: bad argument");
  dim3 grid((unsigned)pairs, (F + 255) / 256);
  if (f32) PRL_CUDA(launch_pdl(moe_glu_kernel<float>, grid, dim3(256), (size_t)0, (cudaStream_t)st, gate_up, ld, F, perm, wsel, limit, beta, (float*)out));
  else PRL_CUDA(launch_pdl(moe_glu_kernel<bf16>, grid, dim3(256), (size_t)0, (cudaStream_t)st, gate_up, ld, F, perm, wsel, limit, beta, (bf16*)out));
  PRL_LAUNCH_CHECK();
  return PRL_OK;
}

// Gated expert activation with the pair's weight on the expert's OUTPUT: out = silu(gate) * up * (wsel * wscale).
extern "C" int prl_moe_glu_out(const float* gate_up, int64_t ld, int64_t pairs, int32_t F, const int32_t* perm,
                               const float* wsel, float wscale, void* out, int32_t f32, prl_stream_t st) {
  PRL_CHECK_ARG(gate_up && perm && wsel && out && pairs >= 1 && F >= 1 && ld >= 2 * (int64_t)F, "prl_moe_glu_out: bad argument");
  dim3 grid((unsigned)pairs, (F + 255) / 256);
  if (f32) PRL_CUDA(launch_pdl(moe_glu_out_kernel<float>, grid, dim3(256), (size_t)0, (cudaStream_t)st, gate_up, ld, F, perm, wsel, wscale, (float*)out));
  else PRL_CUDA(launch_pdl(moe_glu_out_kernel<bf16>, grid, dim3(256), (size_t)0, (cudaStream_t)st, gate_up, ld, F, perm, wsel, wscale, (bf16*)out));
  PRL_LAUNCH_CHECK();
  return PRL_OK;
}
