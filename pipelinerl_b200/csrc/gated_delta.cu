// The gated delta rule of the hybrid decoders, from the input projection to the normed and gated read-out:
//
//     c   = silu(causal convolution of q | k | v),  q = c_q / |c_q| * dk^(-1/2),  k = c_k / |c_k|        (unit length per head)
//     b_t = sigmoid(Z_b),   g_t = exp(-exp(A_log) softplus(Z_a + dt_bias))                              (per value head)
//     S  <- g_t S;   d_t = b_t (v_t - S^T k_t);   S <- S + k_t d_t^T;   o_t = S^T q_t
//     y_t = o_t / rms(o_t) * gain * silu(Z_g)
//
// with `kh` q / k heads serving `heads` value heads.  Everything is fp32; only y is rounded to the operand type.  State:
// [slot][head][dv][dk] (a column's key channels contiguous, the layout of delta_scan.cu), convolution inputs
// [slot][channel][taps - 1], oldest first.
//
// Two paths.
//
// 1. prl_gated_delta_step: segments of one token (a decode step), ONE kernel.  A CTA owns a (segment, q / k head) with all
//    its value heads: it runs the convolution of its channels, shifts their state, forms the unit vectors once, and then
//    passes over the matrix states, each column spread over eight lanes, 64 floats of state per thread in flight.
//
// 2. prl_gated_delta_split: long portions, cut into pieces of up to 64 tokens.  With G_t the product of the decays from the
//    piece's start to t, a piece with incoming state S_0 obeys
//        (I + A) D = b * (V - G * (K S_0)),       A_ts = b_t (G_t / G_s) (k_t . k_s) for s < t
//        O = G * (Q S_0) + E D,                   E_ts = (G_t / G_s) (q_t . k_s) for s <= t
//        S_end = G_end S_0 + (K * (G_end / G))^T D
//    so that D = U - W S_0 with U = (I + A)^(-1) (b * V), W = (I + A)^(-1) (b * G * K).  Four kernels: the front end
//    (convolution, unit vectors, gates); per piece and head A, E and, by forward substitution with two columns per thread, U
//    and W; the walk over the pieces of a segment, which only carries S (two products per piece, a tile of 16 value columns per
//    CTA) and leaves D and every piece's S_0; the read-out, per piece and head again, with the head norm and the gate.  All
//    products are register-blocked fp32 FMAs on the CUDA cores; the piece kernel issues two per instruction (fma.rn.f32x2), on
//    pairs of neighbouring channels or columns.  Decays enter as differences of running sums of logarithms, which are never
//    positive, so nothing overflows.
#include "prl_common.cuh"
#include <math.h>

namespace prl {
namespace {

constexpr int kThreads = 256;
constexpr int kPieceMax = 64;      // tokens per piece
constexpr int kWalkCols = 16;      // value columns per CTA of the walk
constexpr int kOutCols = 128;      // value columns per pass of the read-out

template <typename T> __device__ __forceinline__ void put(T* p, float v);
template <> __device__ __forceinline__ void put<float>(float* p, float v) { *p = v; }
template <> __device__ __forceinline__ void put<__nv_bfloat16>(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float silu_f(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float log_decay(float A_log, float z) {       // -exp(A_log) softplus(z)
  return -expf(A_log) * (z > 20.f ? z : log1pf(expf(z)));
}
__device__ __forceinline__ void cp4z(float* dst, const float* src, int bytes) {
  const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(d), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void cp16z(float* dst, const float* src, int bytes) {
  const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ float4 lds4(const float* p) { return *reinterpret_cast<const float4*>(p); }

// two fp32 numbers in a 64-bit register
typedef unsigned long long pair_t;
__device__ __forceinline__ pair_t fma2(pair_t a, pair_t b, pair_t c) {
  pair_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ pair_t pack2(float x, float y) {
  pair_t d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(x), "f"(y));
  return d;
}
__device__ __forceinline__ float2 unpack2(pair_t a) {
  float2 v;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(v.x), "=f"(v.y) : "l"(a));
  return v;
}
__device__ __forceinline__ float sum2(pair_t a) { const float2 v = unpack2(a); return v.x + v.y; }
__device__ __forceinline__ ulonglong2 ldp(const float* p) { return *reinterpret_cast<const ulonglong2*>(p); }

// rows x cols floats (row stride ld_src) into shared rows of stride ld_dst; rows from `live` on and columns from `cols` to
// `cols_pad` are zero.  `vec`: every source row starts on a 16-byte boundary and cols is a multiple of four.
__device__ __forceinline__ void stage_tile(float* dst, int ld_dst, const float* src, int64_t ld_src, int rows, int live, int cols,
                                           int cols_pad, bool vec) {
  if (vec) {                       // a thread keeps its column and steps over the rows
    const int per = cols_pad / 4, step = blockDim.x / per, c = threadIdx.x % per * 4;
    int r = threadIdx.x / per;
    if (r < step) {
      const float* p = src + r * ld_src + c;
      float* d = dst + r * ld_dst + c;
      for (; r < rows; r += step, p += step * ld_src, d += step * ld_dst) {
        const bool on = r < live && c < cols;
        cp16z(d, on ? p : src, on ? 16 : 0);
      }
    }
  } else {
    for (int i = threadIdx.x; i < rows * cols_pad; i += blockDim.x) {
      const int r = i / cols_pad, c = i - r * cols_pad;
      const bool on = r < live && c < cols;
      cp4z(dst + r * ld_dst + c, src + (on ? r * ld_src + c : 0), on ? 4 : 0);
    }
  }
}

// ---- 1. one token per segment -------------------------------------------------------------------------------------------
struct StepArgs {
  const float* P;             // projection rows: q | k | v at off, logits of beta (off_b) and of the decay (off_a), gate (off_g)
  int64_t ldp;
  int off, off_b, off_a, off_g;
  const float* conv_w;        // [channels][taps]
  int taps;
  const float* A_log;
  const float* dt_bias;
  float unit_eps;
  const float* gain;          // [dv]
  float eps;
  int heads, kh, dk, dv;
  const int32_t* seg_start;
  const int32_t* seg_len;
  const int32_t* seg_slot;
  float* conv_state;
  float* state;
  void* out;                  // [row][heads * dv]
};

// blockDim = 256 * (value heads in flight, 1 or 2); R float4 of a column per lane, eight lanes per column; VEC: dk % 4 == 0
template <typename T, int R, bool VEC>
__global__ void __launch_bounds__(512) gated_delta_step_kernel(StepArgs a) {
  pdl_wait();
  constexpr int CPT = R >= 8 ? 2 : 4;             // columns per thread and pass
  constexpr int dkp = 32 * R;                     // padded key size
  extern __shared__ __align__(16) float sm[];
  const int seg = blockIdx.y, kvh = blockIdx.x;
  if (a.seg_len[seg] != 1) return;                // an idle slot
  const int slot = a.seg_slot[seg];
  const int64_t row = a.seg_start[seg];
  const int rep = a.heads / a.kh, dk = a.dk, dv = a.dv, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int groups = blockDim.x >> 8;
  float* qs = sm;                                 // [dkp]
  float* ks = qs + dkp;                           // [dkp]
  float* os = ks + dkp;                           // [groups][dv]
  float* vs = os + groups * dv;                   // [rep * dv]
  __shared__ float red[16], unit[2];
  const float* p = a.P + row * a.ldp;
  const int ch = 2 * a.kh * dk + a.heads * dv, keep = a.taps - 1;
  const int grp = tid >> 8, t = tid & 255, cg = t >> 3, l8 = t & 7;
  float4 S[CPT][R];
  auto load = [&](const float* S0, int col0) {    // columns col0 + cg + 32 u of a head's state
#pragma unroll
    for (int u = 0; u < CPT; ++u) {
      const int col = col0 + cg + 32 * u;
      const float* s = S0 + (int64_t)col * dk;
#pragma unroll
      for (int j = 0; j < R; ++j) {
        const int i = 4 * (l8 + 8 * j);
        if (VEC) S[u][j] = (col < dv && i < dk) ? *reinterpret_cast<const float4*>(s + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        else {
          const bool in = col < dv;
          S[u][j] = make_float4(in && i < dk ? s[i] : 0.f, in && i + 1 < dk ? s[i + 1] : 0.f, in && i + 2 < dk ? s[i + 2] : 0.f,
                                in && i + 3 < dk ? s[i + 3] : 0.f);
        }
      }
    }
  };
  // the first states are on their way while the convolution runs
  if (grp < rep) load(a.state + ((int64_t)slot * a.heads + kvh * rep + grp) * dv * dk, 0);
  for (int i = tid; i < 2 * (dkp - dk); i += blockDim.x) (i < dkp - dk ? qs + dk + i : ks + dk + i - (dkp - dk))[0] = 0.f;
  for (int i = tid; i < 2 * dk + rep * dv; i += blockDim.x) {
    const int c = i < dk ? kvh * dk + i : i < 2 * dk ? a.kh * dk + kvh * dk + i - dk : 2 * a.kh * dk + kvh * rep * dv + i - 2 * dk;
    const float cur = p[a.off + c];
    const float* w = a.conv_w + (int64_t)c * a.taps;
    float* st = a.conv_state + ((int64_t)slot * ch + c) * keep;
    float acc = 0.f;
    for (int j = 0; j < keep; ++j) {              // oldest first
      const float in = st[j];
      acc = fmaf(w[j], in, acc);
      if (j > 0) st[j - 1] = in;
    }
    if (keep > 0) st[keep - 1] = cur;
    const float v = silu_f(fmaf(w[keep], cur, acc));
    (i < dk ? qs + i : i < 2 * dk ? ks + i - dk : vs + i - 2 * dk)[0] = v;
  }
  __syncthreads();
  if (warp < 2) {
    const float* u = warp ? ks : qs;
    float ss = 0.f;
    for (int i = lane; i < dk; i += 32) ss = fmaf(u[i], u[i], ss);
    ss = warp_sum(ss);
    if (lane == 0) unit[warp] = (warp ? 1.f : 1.f / sqrtf((float)dk)) / sqrtf(ss + a.unit_eps);
  }
  __syncthreads();
  for (int i = tid; i < dk; i += blockDim.x) { qs[i] *= unit[0]; ks[i] *= unit[1]; }
  __syncthreads();
  for (int r0 = 0; r0 < rep; r0 += groups) {
    const bool on = r0 + grp < rep;               // uniform over the group's warps
    const int head = kvh * rep + r0 + grp;
    float* o = os + grp * dv;
    if (on) {
      const float beta = sigmoid_f(p[a.off_b + head]);
      const float g = expf(log_decay(a.A_log[head], p[a.off_a + head] + a.dt_bias[head]));
      float* S0 = a.state + ((int64_t)slot * a.heads + head) * dv * dk;
      for (int col0 = 0; col0 < dv; col0 += 32 * CPT) {
        if (r0 + col0 > 0) load(S0, col0);
        float dot[CPT], rd[CPT];
#pragma unroll
        for (int u = 0; u < CPT; ++u) { dot[u] = 0.f; rd[u] = 0.f; }
#pragma unroll
        for (int j = 0; j < R; ++j) {
          const float4 k = lds4(ks + 4 * (l8 + 8 * j));
#pragma unroll
          for (int u = 0; u < CPT; ++u) {
            S[u][j].x *= g; S[u][j].y *= g; S[u][j].z *= g; S[u][j].w *= g;
            dot[u] = fmaf(k.x, S[u][j].x, dot[u]); dot[u] = fmaf(k.y, S[u][j].y, dot[u]);
            dot[u] = fmaf(k.z, S[u][j].z, dot[u]); dot[u] = fmaf(k.w, S[u][j].w, dot[u]);
          }
        }
#pragma unroll
        for (int m = 1; m < 8; m <<= 1)
#pragma unroll
          for (int u = 0; u < CPT; ++u) dot[u] += __shfl_xor_sync(0xffffffffu, dot[u], m);
#pragma unroll
        for (int u = 0; u < CPT; ++u) {
          const int col = col0 + cg + 32 * u;
          dot[u] = beta * ((col < dv ? vs[(r0 + grp) * dv + col] : 0.f) - dot[u]);
        }
#pragma unroll
        for (int j = 0; j < R; ++j) {
          const float4 k = lds4(ks + 4 * (l8 + 8 * j)), q = lds4(qs + 4 * (l8 + 8 * j));
#pragma unroll
          for (int u = 0; u < CPT; ++u) {
            S[u][j].x = fmaf(k.x, dot[u], S[u][j].x); S[u][j].y = fmaf(k.y, dot[u], S[u][j].y);
            S[u][j].z = fmaf(k.z, dot[u], S[u][j].z); S[u][j].w = fmaf(k.w, dot[u], S[u][j].w);
            rd[u] = fmaf(q.x, S[u][j].x, rd[u]); rd[u] = fmaf(q.y, S[u][j].y, rd[u]);
            rd[u] = fmaf(q.z, S[u][j].z, rd[u]); rd[u] = fmaf(q.w, S[u][j].w, rd[u]);
          }
        }
#pragma unroll
        for (int u = 0; u < CPT; ++u) {
          const int col = col0 + cg + 32 * u;
          float* s = S0 + (int64_t)col * dk;
#pragma unroll
          for (int j = 0; j < R; ++j) {
            const int i = 4 * (l8 + 8 * j);
            if (col >= dv) continue;
            if (VEC) { if (i < dk) *reinterpret_cast<float4*>(s + i) = S[u][j]; }
            else {
              if (i < dk) s[i] = S[u][j].x;
              if (i + 1 < dk) s[i + 1] = S[u][j].y;
              if (i + 2 < dk) s[i + 2] = S[u][j].z;
              if (i + 3 < dk) s[i + 3] = S[u][j].w;
            }
          }
        }
#pragma unroll
        for (int m = 1; m < 8; m <<= 1)
#pragma unroll
          for (int u = 0; u < CPT; ++u) rd[u] += __shfl_xor_sync(0xffffffffu, rd[u], m);
#pragma unroll
        for (int u = 0; u < CPT; ++u) {
          const int col = col0 + cg + 32 * u;
          if (l8 == 0 && col < dv) o[col] = rd[u];
        }
      }
    }
    __syncthreads();
    float ss = 0.f;
    if (on)
      for (int c = t; c < dv; c += 256) ss = fmaf(o[c], o[c], ss);
    ss = warp_sum(ss);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    if (on) {
      float tot = 0.f;
      for (int w = 0; w < 8; ++w) tot += red[8 * grp + w];
      const float inv = 1.f / sqrtf(tot / (float)dv + a.eps);
      T* y = reinterpret_cast<T*>(a.out) + (row * a.heads + head) * dv;
      const float* z = p + a.off_g + head * dv;
      for (int c = t; c < dv; c += 256) put(y + c, o[c] * inv * a.gain[c] * silu_f(z[c]));
    }
    __syncthreads();                              // os and red are written again by the next pass
  }
}

// ---- 2. pieces -------------------------------------------------------------------------------------------------------------
struct SplitArgs {
  const float* P;
  int64_t ldp;
  int off, off_b, off_a, off_g;
  const float* conv_w;
  int taps;
  const float* A_log;
  const float* dt_bias;
  float unit_eps;
  const float* gain;
  float eps;
  int heads, kh, dk, dv, vec;
  const int32_t* row_slot;
  const int32_t* row_back;
  const int32_t* seg_start;
  const int32_t* seg_len;
  const int32_t* seg_slot;
  const int32_t* seg_sub0;
  const int32_t* seg_nsub;
  const int32_t* sub_start;
  const int32_t* sub_len;
  float* C;                   // [row][channels]: unit q (times dk^(-1/2)) | unit k | v
  float* gates;               // [row][2 * heads]: log decay (later its running sum within the piece) | beta
  float* W;                   // [row][heads * dk]
  float* E;                   // [row][heads * 64]
  float* D;                   // [row][heads * dv]: U, then D (dv > 128: then the read-out)
  float* S0;                  // [piece][heads][dk][dv]
  float* conv_state;
  float* state;
  void* out;                  // [row][heads * dv]
};

// Convolution, unit vectors and gates of one row; a warp per head of q, of k and of v.
__global__ void __launch_bounds__(kThreads) gated_delta_front_kernel(SplitArgs a) {
  pdl_wait();
  const int64_t row = blockIdx.x;
  const int slot = a.row_slot[row];
  if (slot < 0) return;
  const int back = a.row_back[row], warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int dk = a.dk, dv = a.dv, keep = a.taps - 1, ch = 2 * a.kh * dk + a.heads * dv;
  const float* p = a.P + row * a.ldp;
  auto conv = [&](int c) {
    const float* w = a.conv_w + (int64_t)c * a.taps;
    const float* st = a.conv_state + ((int64_t)slot * ch + c) * keep;
    float acc = 0.f;
    for (int k = keep; k >= 0; --k) {             // oldest first
      const float in = k <= back ? p[a.off + c - (int64_t)k * a.ldp] : st[keep - (k - back)];
      acc = fmaf(w[keep - k], in, acc);
    }
    return silu_f(acc);
  };
  float* out = a.C + row * ch;
  for (int h = warp; h < 2 * a.kh + a.heads; h += kThreads / 32) {
    if (h < 2 * a.kh) {
      const int c0 = h * dk;
      float v[8], ss = 0.f;
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const int i = lane + 32 * j;
        v[j] = i < dk ? conv(c0 + i) : 0.f;
        ss = fmaf(v[j], v[j], ss);
      }
      ss = warp_sum(ss);
      const float f = (h < a.kh ? 1.f / sqrtf((float)dk) : 1.f) / sqrtf(ss + a.unit_eps);
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const int i = lane + 32 * j;
        if (i < dk) out[c0 + i] = v[j] * f;
      }
    } else {
      const int c0 = 2 * a.kh * dk + (h - 2 * a.kh) * dv;
      for (int i = lane; i < dv; i += 32) out[c0 + i] = conv(c0 + i);
    }
  }
  for (int h = threadIdx.x; h < a.heads; h += kThreads) {
    a.gates[row * 2 * a.heads + h] = log_decay(a.A_log[h], p[a.off_a + h] + a.dt_bias[h]);
    a.gates[row * 2 * a.heads + a.heads + h] = sigmoid_f(p[a.off_b + h]);
  }
}

// The same for head sizes of a multiple of four and TAPS taps: a warp runs one head over kFrontRows consecutive rows, four
// channels per lane, so that a row's inputs are read once and serve the taps of the rows behind it from registers.
constexpr int kFrontRows = 4;
template <int TAPS>
__global__ void __launch_bounds__(kThreads) gated_delta_front_tile_kernel(SplitArgs a, int n_rows) {
  pdl_wait();
  constexpr int keep = TAPS - 1, RT = kFrontRows;
  const int row0 = blockIdx.x * RT, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int dk = a.dk, dv = a.dv, H = a.heads, ch = 2 * a.kh * dk + H * dv;
  int slot[RT], back[RT];
#pragma unroll
  for (int r = 0; r < RT; ++r) {
    slot[r] = row0 + r < n_rows ? a.row_slot[row0 + r] : -1;
    back[r] = row0 + r < n_rows ? a.row_back[row0 + r] : 0;
  }
  const int h = blockIdx.y * (kThreads / 32) + warp;
  if (h < 2 * a.kh + H) {
    const bool unit = h < 2 * a.kh;
    const int c0 = unit ? h * dk : 2 * a.kh * dk + (h - 2 * a.kh) * dv, groups = (unit ? dk : dv) / 4;
    const float* p = a.P + (int64_t)row0 * a.ldp + a.off;
    for (int g0 = 0; g0 < groups; g0 += 64) {             // a head with unit length has at most 64 groups: one pass
      float4 v[2][RT];
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const int g = g0 + lane + 32 * u;
        if (g >= groups) {
#pragma unroll
          for (int r = 0; r < RT; ++r) v[u][r] = make_float4(0.f, 0.f, 0.f, 0.f);
          continue;
        }
        const int c = c0 + 4 * g;
        float4 x[keep + RT];                              // inputs of rows row0 - keep .. row0 + RT - 1 (of this batch only)
#pragma unroll
        for (int j = 0; j < keep + RT; ++j) {
          const bool in = j < keep ? keep - j <= back[0] : row0 + j - keep < n_rows;
          x[j] = in ? *reinterpret_cast<const float4*>(p + (int64_t)(j - keep) * a.ldp + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
        float w[4][TAPS];
#pragma unroll
        for (int e = 0; e < 4; ++e)
#pragma unroll
          for (int k = 0; k < TAPS; ++k) w[e][k] = a.conv_w[(int64_t)(c + e) * TAPS + k];
#pragma unroll
        for (int r = 0; r < RT; ++r) {
          float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
          if (slot[r] >= 0) {
#pragma unroll
            for (int k = keep; k >= 0; --k) {             // oldest first
              float4 in = x[keep + r - k];
              if (k > back[r]) {                          // before this batch: the carried inputs
                const float* st = a.conv_state + ((int64_t)slot[r] * ch + c) * keep + keep - (k - back[r]);
                in = make_float4(st[0], st[keep], st[2 * keep], st[3 * keep]);
              }
              acc.x = fmaf(w[0][keep - k], in.x, acc.x); acc.y = fmaf(w[1][keep - k], in.y, acc.y);
              acc.z = fmaf(w[2][keep - k], in.z, acc.z); acc.w = fmaf(w[3][keep - k], in.w, acc.w);
            }
          }
          v[u][r] = make_float4(silu_f(acc.x), silu_f(acc.y), silu_f(acc.z), silu_f(acc.w));
        }
      }
#pragma unroll
      for (int r = 0; r < RT; ++r) {
        float f = 1.f;
        if (unit) {
          float ss = 0.f;
#pragma unroll
          for (int u = 0; u < 2; ++u)
            ss += v[u][r].x * v[u][r].x + v[u][r].y * v[u][r].y + v[u][r].z * v[u][r].z + v[u][r].w * v[u][r].w;
          f = (h < a.kh ? 1.f / sqrtf((float)dk) : 1.f) / sqrtf(warp_sum(ss) + a.unit_eps);
        }
        if (slot[r] < 0) continue;
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          const int g = g0 + lane + 32 * u;
          if (g < groups)
            *reinterpret_cast<float4*>(a.C + (int64_t)(row0 + r) * ch + c0 + 4 * g) =
                make_float4(v[u][r].x * f, v[u][r].y * f, v[u][r].z * f, v[u][r].w * f);
        }
      }
    }
  }
  if (blockIdx.y == 0)
    for (int i = threadIdx.x; i < RT * H; i += kThreads) {
      const int r = i / H, hh = i - r * H;
      const int64_t row = row0 + r;
      if (row >= n_rows || a.row_slot[row] < 0) continue;
      a.gates[row * 2 * H + hh] = log_decay(a.A_log[hh], a.P[row * a.ldp + a.off_a + hh] + a.dt_bias[hh]);
      a.gates[row * 2 * H + H + hh] = sigmoid_f(a.P[row * a.ldp + a.off_b + hh]);
    }
}

// A, E, U and W of one (piece, value head); the running sums of the log decays replace them in `gates`.
// A is kept negated and doubled (each entry as a pair), as the ten 16 x 16 blocks on and below its diagonal: block (b, q) at
// b (b + 1) / 2 + q, entry (column s, row t) at 32 s + 2 t.
constexpr int kPieceThreads = 128;
constexpr int kBlk = 16, kBlkFloats = kBlk * kBlk * 2;
__device__ __forceinline__ int blk_at(int b, int q) { return (b * (b + 1) / 2 + q) * kBlkFloats; }

__global__ void __launch_bounds__(kPieceThreads, 2) gated_delta_piece_kernel(SplitArgs a) {
  pdl_wait();
  extern __shared__ __align__(16) float sm[];
  const int piece = blockIdx.x, head = blockIdx.y, len = a.sub_len[piece];
  const int64_t row0 = a.sub_start[piece];
  const int dk = a.dk, dv = a.dv, H = a.heads, tid = threadIdx.x;
  const int dk4 = (dk + 3) & ~3, ldk = dk4 + 4, ch = 2 * a.kh * dk + H * dv, kvh = head / (H / a.kh);
  float* As = sm;                                 // 10 blocks
  float* Ks = As + 10 * kBlkFloats;               // [64][ldk]
  float* Qs = Ks + kPieceMax * ldk;               // [64][ldk], later X: rows 0 .. 47 of the thread's two columns [48][256]
  __shared__ float cum[kPieceMax], beta[kPieceMax], bg[kPieceMax];      // running log decay, step, step times decay
  const float* C = a.C + row0 * ch;
  stage_tile(Ks, ldk, C + a.kh * dk + kvh * dk, ch, kPieceMax, len, dk, dk4, a.vec);
  stage_tile(Qs, ldk, C + kvh * dk, ch, kPieceMax, len, dk, dk4, a.vec);
  cp_commit();
  if (tid < 32) {                                 // running sums of the log decays, two tokens per lane
    float* gr = a.gates + row0 * 2 * H + head;
    const int t0 = 2 * tid;
    const float l0 = t0 < len ? gr[(int64_t)t0 * 2 * H] : 0.f, l1 = t0 + 1 < len ? gr[(int64_t)(t0 + 1) * 2 * H] : 0.f;
    float s = l0 + l1;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, s, o);
      if (tid >= o) s += v;
    }
    cum[t0] = s - l1;
    cum[t0 + 1] = s;
    beta[t0] = t0 < len ? gr[(int64_t)t0 * 2 * H + H] : 0.f;
    beta[t0 + 1] = t0 + 1 < len ? gr[(int64_t)(t0 + 1) * 2 * H + H] : 0.f;
    bg[t0] = beta[t0] * expf(cum[t0]);
    bg[t0 + 1] = beta[t0 + 1] * expf(cum[t0 + 1]);
    if (t0 < len) gr[(int64_t)t0 * 2 * H] = s - l1;
    if (t0 + 1 < len) gr[(int64_t)(t0 + 1) * 2 * H] = s;
  }
  cp_wait<0>();
  __syncthreads();
  {   // one half of the CTA forms K K^T, the other Q K^T, 8 x 8 entries per thread
    const bool query = tid >= 64;
    const int ty = tid >> 3 & 7, tx = tid & 7;
    const float* rows = query ? Qs : Ks;
    pair_t acc[8][8];
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int j = 0; j <= i; ++j) acc[i][j] = 0ull;
    for (int c = 0; c < dk4; c += 4) {
      ulonglong2 s4[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) s4[j] = ldp(Ks + (tx + 8 * j) * ldk + c);
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const ulonglong2 r4 = ldp(rows + (ty + 8 * i) * ldk + c);
#pragma unroll
        for (int j = 0; j <= i; ++j)              // blocks above the diagonal are not needed
          acc[i][j] = fma2(r4.y, s4[j].y, fma2(r4.x, s4[j].x, acc[i][j]));
      }
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int t = ty + 8 * i;
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const int s = tx + 8 * j;
        const float e = j <= i && s <= t ? expf(cum[t] - cum[s]) * sum2(acc[i][j <= i ? j : 0]) : 0.f;
        if (query) {
          if (t < len) a.E[((row0 + t) * H + head) * kPieceMax + s] = s < len ? e : 0.f;
        } else if (i / 2 >= j / 2) {              // a block on or below the diagonal; rows past the piece have beta = 0
          const float v = s < t ? -beta[t] * e : 0.f;
          *reinterpret_cast<float2*>(As + blk_at(i / 2, j / 2) + 32 * (s & 15) + 2 * (t & 15)) = make_float2(v, v);
        }
      }
    }
  }
  __syncthreads();
  // forward substitution for two neighbouring columns of [b V | b G K] per thread, sixteen rows at a time: the rows done so
  // far come back from shared memory (only the thread itself reads them)
  const float* V = C + 2 * a.kh * dk + head * dv;
  float* X = Qs + 2 * tid;
  for (int col = 2 * tid; col < dv + dk; col += 2 * kPieceThreads) {
    const bool two = col + 1 < dv + dk, same = a.vec;      // vec: dv is even, so both columns are in one matrix
#pragma unroll 1
    for (int b = 0; b < kPieceMax / kBlk; ++b) {
      if (b * kBlk >= len) break;                 // rows past the piece are zero and nobody reads them
      pair_t r[kBlk];
      if (same && col < dv) {
#pragma unroll
        for (int t = 0; t < kBlk; ++t) {
          const int tt = b * kBlk + t;
          const float2 v = tt < len ? *reinterpret_cast<const float2*>(V + (int64_t)tt * ch + col) : make_float2(0.f, 0.f);
          r[t] = pack2(beta[tt] * v.x, beta[tt] * v.y);
        }
      } else {
#pragma unroll
        for (int t = 0; t < kBlk; ++t) {
          const int tt = b * kBlk + t;
          float v[2];
#pragma unroll
          for (int u = 0; u < 2; ++u) {
            const int c = col + u;
            v[u] = c < dv ? (tt < len ? beta[tt] * V[(int64_t)tt * ch + c] : 0.f) : c < dv + dk ? bg[tt] * Ks[tt * ldk + c - dv] : 0.f;
          }
          r[t] = pack2(v[0], v[1]);
        }
      }
#pragma unroll 1
      for (int q = 0; q < b; ++q) {
        const float* blk = As + blk_at(b, q);
#pragma unroll 4
        for (int s = 0; s < kBlk; ++s) {
          const pair_t x = *reinterpret_cast<const pair_t*>(X + (q * kBlk + s) * 2 * kPieceThreads);
#pragma unroll
          for (int t = 0; t < kBlk; t += 2) {
            const ulonglong2 w = ldp(blk + 32 * s + 2 * t);
            r[t] = fma2(w.x, x, r[t]);
            r[t + 1] = fma2(w.y, x, r[t + 1]);
          }
        }
      }
      const float* blk = As + blk_at(b, b);
#pragma unroll
      for (int s = 0; s < kBlk - 1; ++s) {
#pragma unroll
        for (int t = (s + 1) / 2 * 2; t < kBlk; t += 2) {
          const ulonglong2 w = ldp(blk + 32 * s + 2 * t);
          if (t > s) r[t] = fma2(w.x, r[s], r[t]);
          if (t + 1 > s) r[t + 1] = fma2(w.y, r[s], r[t + 1]);
        }
      }
#pragma unroll
      for (int t = 0; t < kBlk; ++t) {
        const int tt = b * kBlk + t;
        if (b + 1 < kPieceMax / kBlk) *reinterpret_cast<pair_t*>(X + tt * 2 * kPieceThreads) = r[t];
        if (tt >= len) continue;
        const float2 v = unpack2(r[t]);
        float* u = a.D + ((row0 + tt) * H + head) * dv;
        float* w = a.W + ((row0 + tt) * H + head) * dk - dv;
        if (same) *reinterpret_cast<float2*>((col < dv ? u : w) + col) = v;
        else {
          (col < dv ? u : w)[col] = v.x;
          if (two) (col + 1 < dv ? u : w)[col + 1] = v.y;
        }
      }
    }
  }
}

// The pieces of a segment in order, for one value head and a tile of 16 value columns: D = U - W S, S <- G S + (K G / G_t)^T D.
// STAGES tiles of (W, K) in shared memory: two when a CTA has its SM alone, one when two CTAs share it.
template <int STAGES>
__global__ void __launch_bounds__(kThreads, 2) gated_delta_walk_kernel(SplitArgs a) {
  pdl_wait();
  extern __shared__ __align__(16) float sm[];
  const int col0 = blockIdx.x * kWalkCols, head = blockIdx.y, seg = blockIdx.z;
  const int np = a.seg_nsub[seg], first = a.seg_sub0[seg], slen = a.seg_len[seg];
  if (np <= 0 || slen <= 0) return;
  const int slot = a.seg_slot[seg];
  const int dk = a.dk, dv = a.dv, H = a.heads, tid = threadIdx.x;
  const int dk4 = (dk + 3) & ~3, ldk = dk4 + 4, ch = 2 * a.kh * dk + H * dv, kvh = head / (H / a.kh);
  constexpr int ldc = kWalkCols + 4;
  const int tile = 2 * kPieceMax * ldk;
  float* bufs = sm;                               // [STAGES]: W [64][ldk] | K [64][ldk]
  float* S = bufs + STAGES * tile;                // [dk4][ldc]
  float* Ds = S + dk4 * ldc;                      // [64][ldc]: D times G_end / G_t
  float* red = Ds + kPieceMax * ldc;              // partial sums: [4][64][16] of W S, then [dk4][16] of the update
  __shared__ float fin[kPieceMax];                // G_end / G_t
  __shared__ float gend;
  // the convolution's last inputs become the segment's state (the front end has read the old ones)
  const int keep = a.taps - 1;
  for (int c = (blockIdx.y * gridDim.x + blockIdx.x) * kThreads + tid; c < ch && keep > 0; c += gridDim.x * gridDim.y * kThreads) {
    float* st = a.conv_state + ((int64_t)slot * ch + c) * keep;
    const int64_t last = (int64_t)a.seg_start[seg] + slen - 1;
    for (int j = 0; j < keep; ++j) {              // ascending: st[j + slen] is still the old input
      const int e = keep - 1 - j;
      st[j] = e < slen ? a.P[(last - e) * a.ldp + a.off + c] : st[j + slen];
    }
  }
  float* state = a.state + ((int64_t)slot * H + head) * dv * dk;
  for (int i = tid; i < kWalkCols * dk4; i += kThreads) {
    const int c = i / dk4, k = i - c * dk4;
    S[k * ldc + c] = (col0 + c < dv && k < dk) ? state[(int64_t)(col0 + c) * dk + k] : 0.f;
  }
  auto stage = [&](int i) {
    if (i < np) {
      const int64_t r0 = a.sub_start[first + i];
      const int len = a.sub_len[first + i];
      float* b = bufs + (i % STAGES) * tile;
      stage_tile(b, ldk, a.W + (r0 * H + head) * dk, (int64_t)H * dk, kPieceMax, len, dk, dk4, a.vec);
      stage_tile(b + kPieceMax * ldk, ldk, a.C + r0 * ch + a.kh * dk + kvh * dk, ch, kPieceMax, len, dk, dk4, a.vec);
    }
    cp_commit();
  };
  if (STAGES > 1) stage(0);
  const int cg = tid & 3;                         // columns 4 cg .. 4 cg + 3 in every role of the thread
  // W S: two warps per quarter of the key channels, rows rg + 16 m
  const int slice = tid >> 6, rg = tid >> 2 & 15, k_len = (dk4 + 15) / 16 * 4;
  const int k_lo = min(dk4, slice * k_len), k_hi = min(dk4, k_lo + k_len);
  // D: row dt
  const int dt = tid >> 2;
  // update: half of the rows, key channels 4 kg .. and 128 + 4 kg ..
  const int half = tid >> 7, kg = tid >> 2 & 31;
  const bool vec_col = a.vec && col0 + 4 * cg < dv;
  for (int i = 0; i < np; ++i) {
    const int64_t r0 = a.sub_start[first + i];
    const int len = a.sub_len[first + i];
    if (STAGES > 1) { stage(i + 1); cp_wait<1>(); } else { stage(i); cp_wait<0>(); }
    const float* Ws = bufs + (i % STAGES) * tile;
    const float* Kt = Ws + kPieceMax * ldk;
    if (tid < kPieceMax) {
      const float* gr = a.gates + r0 * 2 * H + head;
      const float end = gr[(int64_t)(len - 1) * 2 * H];
      fin[tid] = tid < len ? expf(end - gr[(int64_t)tid * 2 * H]) : 0.f;
      if (tid == 0) gend = expf(end);
    }
    float* Drow = a.D + ((r0 + dt) * H + head) * dv + col0 + 4 * cg;
    float4 d = make_float4(0.f, 0.f, 0.f, 0.f);                       // U of row dt
    if (dt < len) {
      if (vec_col) d = *reinterpret_cast<const float4*>(Drow);
      else {
        const int left = dv - col0 - 4 * cg;
        if (left > 0) d.x = Drow[0];
        if (left > 1) d.y = Drow[1];
        if (left > 2) d.z = Drow[2];
        if (left > 3) d.w = Drow[3];
      }
    }
    __syncthreads();
    {
      float4 u[4];
#pragma unroll
      for (int m = 0; m < 4; ++m) u[m] = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int k = k_lo; k < k_hi; k += 4) {
        const float4 s0 = lds4(S + k * ldc + 4 * cg), s1 = lds4(S + (k + 1) * ldc + 4 * cg), s2 = lds4(S + (k + 2) * ldc + 4 * cg),
                     s3 = lds4(S + (k + 3) * ldc + 4 * cg);
#pragma unroll
        for (int m = 0; m < 4; ++m) {
          const float4 q = lds4(Ws + (rg + 16 * m) * ldk + k);
          u[m].x = fmaf(q.x, s0.x, u[m].x); u[m].y = fmaf(q.x, s0.y, u[m].y); u[m].z = fmaf(q.x, s0.z, u[m].z); u[m].w = fmaf(q.x, s0.w, u[m].w);
          u[m].x = fmaf(q.y, s1.x, u[m].x); u[m].y = fmaf(q.y, s1.y, u[m].y); u[m].z = fmaf(q.y, s1.z, u[m].z); u[m].w = fmaf(q.y, s1.w, u[m].w);
          u[m].x = fmaf(q.z, s2.x, u[m].x); u[m].y = fmaf(q.z, s2.y, u[m].y); u[m].z = fmaf(q.z, s2.z, u[m].z); u[m].w = fmaf(q.z, s2.w, u[m].w);
          u[m].x = fmaf(q.w, s3.x, u[m].x); u[m].y = fmaf(q.w, s3.y, u[m].y); u[m].z = fmaf(q.w, s3.z, u[m].z); u[m].w = fmaf(q.w, s3.w, u[m].w);
        }
      }
#pragma unroll
      for (int m = 0; m < 4; ++m) *reinterpret_cast<float4*>(red + (slice * kPieceMax + rg + 16 * m) * kWalkCols + 4 * cg) = u[m];
    }
    {   // S at the piece's start, for the read-out
      float* dst = a.S0 + ((int64_t)(first + i) * H + head) * dk * dv + col0 + 4 * cg;
      for (int k = tid >> 2; k < dk; k += kThreads / 4) {
        const float4 v = lds4(S + k * ldc + 4 * cg);
        float* p = dst + (int64_t)k * dv;
        if (vec_col) *reinterpret_cast<float4*>(p) = v;
        else {
          const int left = dv - col0 - 4 * cg;
          if (left > 0) p[0] = v.x;
          if (left > 1) p[1] = v.y;
          if (left > 2) p[2] = v.z;
          if (left > 3) p[3] = v.w;
        }
      }
    }
    __syncthreads();
#pragma unroll
    for (int q = 0; q < 4; ++q) {
      const float4 v = lds4(red + (q * kPieceMax + dt) * kWalkCols + 4 * cg);
      d.x -= v.x; d.y -= v.y; d.z -= v.z; d.w -= v.w;
    }
    if (dt < len) {
      if (vec_col) *reinterpret_cast<float4*>(Drow) = d;
      else {
        const int left = dv - col0 - 4 * cg;
        if (left > 0) Drow[0] = d.x;
        if (left > 1) Drow[1] = d.y;
        if (left > 2) Drow[2] = d.z;
        if (left > 3) Drow[3] = d.w;
      }
    }
    const float f = fin[dt];
    *reinterpret_cast<float4*>(Ds + dt * ldc + 4 * cg) = make_float4(d.x * f, d.y * f, d.z * f, d.w * f);
    __syncthreads();                              // D complete, every read of the old S and of the partial sums done
    const float ge = gend;
    float4 acc[2][4];                             // two passes of 128 key channels
#pragma unroll
    for (int p = 0; p < 2; ++p) {
      const int k0 = 4 * kg + 128 * p;
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[p][e] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (k0 >= dk4) continue;
#pragma unroll 8
      for (int t = half * (kPieceMax / 2); t < (half + 1) * (kPieceMax / 2); ++t) {
        const float4 kv = lds4(Kt + t * ldk + k0), v = lds4(Ds + t * ldc + 4 * cg);
        acc[p][0].x = fmaf(kv.x, v.x, acc[p][0].x); acc[p][0].y = fmaf(kv.x, v.y, acc[p][0].y); acc[p][0].z = fmaf(kv.x, v.z, acc[p][0].z); acc[p][0].w = fmaf(kv.x, v.w, acc[p][0].w);
        acc[p][1].x = fmaf(kv.y, v.x, acc[p][1].x); acc[p][1].y = fmaf(kv.y, v.y, acc[p][1].y); acc[p][1].z = fmaf(kv.y, v.z, acc[p][1].z); acc[p][1].w = fmaf(kv.y, v.w, acc[p][1].w);
        acc[p][2].x = fmaf(kv.z, v.x, acc[p][2].x); acc[p][2].y = fmaf(kv.z, v.y, acc[p][2].y); acc[p][2].z = fmaf(kv.z, v.z, acc[p][2].z); acc[p][2].w = fmaf(kv.z, v.w, acc[p][2].w);
        acc[p][3].x = fmaf(kv.w, v.x, acc[p][3].x); acc[p][3].y = fmaf(kv.w, v.y, acc[p][3].y); acc[p][3].z = fmaf(kv.w, v.z, acc[p][3].z); acc[p][3].w = fmaf(kv.w, v.w, acc[p][3].w);
      }
      if (half)
#pragma unroll
        for (int e = 0; e < 4; ++e) *reinterpret_cast<float4*>(red + (k0 + e) * kWalkCols + 4 * cg) = acc[p][e];
    }
    __syncthreads();
    if (!half)
#pragma unroll
      for (int p = 0; p < 2; ++p) {
        const int k0 = 4 * kg + 128 * p;
        if (k0 >= dk4) continue;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          float4* sp = reinterpret_cast<float4*>(S + (k0 + e) * ldc + 4 * cg);
          const float4 o = lds4(red + (k0 + e) * kWalkCols + 4 * cg), v = *sp;
          *sp = make_float4(fmaf(ge, v.x, acc[p][e].x + o.x), fmaf(ge, v.y, acc[p][e].y + o.y), fmaf(ge, v.z, acc[p][e].z + o.z),
                            fmaf(ge, v.w, acc[p][e].w + o.w));
        }
      }
    __syncthreads();                              // the next piece's copies and gates overwrite what was read here
  }
  cp_wait<0>();
  for (int i = tid; i < kWalkCols * dk; i += kThreads) {
    const int c = i / dk, k = i - c * dk;
    if (col0 + c < dv) state[(int64_t)(col0 + c) * dk + k] = S[k * ldc + c];
  }
}

// O = G * (Q S_0) + E D of one (piece, value head), 128 value columns per pass; NORM (dv <= 128): the head norm, the gain and
// the gate, into `out`; otherwise the raw read-out replaces D.
template <typename T, bool NORM>
__global__ void __launch_bounds__(kThreads, 2) gated_delta_read_kernel(SplitArgs a) {
  pdl_wait();
  extern __shared__ __align__(16) float sm[];
  constexpr int kStep = 32, lda = kStep + 4, ldb = kOutCols + 4;
  const int piece = blockIdx.x, head = blockIdx.y, col0 = blockIdx.z * kOutCols, len = a.sub_len[piece];
  const int64_t row0 = a.sub_start[piece];
  const int dk = a.dk, dv = a.dv, H = a.heads, tid = threadIdx.x, ch = 2 * a.kh * dk + H * dv, kvh = head / (H / a.kh);
  const int nc = min(kOutCols, dv - col0);        // live columns
  float* As = sm;                                 // [2][64][lda]
  float* Bs = As + 2 * kPieceMax * lda;           // [2][32][ldb]
  const int n1 = (dk + kStep - 1) / kStep, n2 = (len + kStep - 1) / kStep;
  auto stage = [&](int i) {
    if (i < n1 + n2) {
      float* as = As + (i & 1) * kPieceMax * lda;
      float* bs = Bs + (i & 1) * kStep * ldb;
      if (i < n1) {                               // Q rows, rows of S_0
        const int k0 = i * kStep, nk = min(kStep, dk - k0);
        stage_tile(as, lda, a.C + row0 * ch + kvh * dk + k0, ch, kPieceMax, len, nk, kStep, a.vec);
        stage_tile(bs, ldb, a.S0 + (((int64_t)piece * H + head) * dk + k0) * dv + col0, dv, kStep, nk, nc, kOutCols, a.vec);
      } else {                                    // rows of E, rows of D
        const int s0 = (i - n1) * kStep, ns = min(kStep, len - s0);
        stage_tile(as, lda, a.E + (row0 * H + head) * kPieceMax + s0, (int64_t)H * kPieceMax, kPieceMax, len, kStep, kStep, true);
        stage_tile(bs, ldb, a.D + ((row0 + s0) * H + head) * dv + col0, (int64_t)H * dv, kStep, ns, nc, kOutCols, a.vec);
      }
    }
    cp_commit();
  };
  const int ty = tid >> 4, tx = tid & 15;         // rows ty + 16 m, columns 4 tx .. and 64 + 4 tx ..
  float acc[4][8];
#pragma unroll
  for (int m = 0; m < 4; ++m)
#pragma unroll
    for (int c = 0; c < 8; ++c) acc[m][c] = 0.f;
  float up[4];                                    // G_t
#pragma unroll
  for (int m = 0; m < 4; ++m) {
    const int t = ty + 16 * m;
    up[m] = t < len ? expf(a.gates[(row0 + t) * 2 * H + head]) : 0.f;
  }
  stage(0);
  for (int i = 0; i < n1 + n2; ++i) {
    stage(i + 1);                                 // its buffer was read one step ago
    cp_wait<1>();
    __syncthreads();
    if (i == n1)
#pragma unroll
      for (int m = 0; m < 4; ++m)
#pragma unroll
        for (int c = 0; c < 8; ++c) acc[m][c] *= up[m];
    const float* as = As + (i & 1) * kPieceMax * lda;
    const float* bs = Bs + (i & 1) * kStep * ldb;
#pragma unroll
    for (int k = 0; k < kStep; k += 4) {
      float4 q[4];
#pragma unroll
      for (int m = 0; m < 4; ++m) q[m] = lds4(as + (ty + 16 * m) * lda + k);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float4 b0 = lds4(bs + (k + e) * ldb + 4 * tx), b1 = lds4(bs + (k + e) * ldb + 64 + 4 * tx);
#pragma unroll
        for (int m = 0; m < 4; ++m) {
          const float w = e == 0 ? q[m].x : e == 1 ? q[m].y : e == 2 ? q[m].z : q[m].w;
          acc[m][0] = fmaf(w, b0.x, acc[m][0]); acc[m][1] = fmaf(w, b0.y, acc[m][1]); acc[m][2] = fmaf(w, b0.z, acc[m][2]); acc[m][3] = fmaf(w, b0.w, acc[m][3]);
          acc[m][4] = fmaf(w, b1.x, acc[m][4]); acc[m][5] = fmaf(w, b1.y, acc[m][5]); acc[m][6] = fmaf(w, b1.z, acc[m][6]); acc[m][7] = fmaf(w, b1.w, acc[m][7]);
        }
      }
    }
    __syncthreads();
  }
  cp_wait<0>();
#pragma unroll
  for (int m = 0; m < 4; ++m) {
    const int t = ty + 16 * m;
    if constexpr (NORM) {
      float ss = 0.f;                             // columns past dv are zero
#pragma unroll
      for (int c = 0; c < 8; ++c) ss = fmaf(acc[m][c], acc[m][c], ss);
#pragma unroll
      for (int o = 1; o < 16; o <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      if (t >= len) continue;
      const float inv = 1.f / sqrtf(ss / (float)dv + a.eps);
      const float* z = a.P + (row0 + t) * a.ldp + a.off_g + head * dv;
      T* y = reinterpret_cast<T*>(a.out) + ((row0 + t) * H + head) * dv;
#pragma unroll
      for (int c = 0; c < 8; ++c) {
        const int col = (c >> 2) * 64 + 4 * tx + (c & 3);
        if (col < nc) put(y + col, acc[m][c] * inv * a.gain[col] * silu_f(z[col]));
      }
    } else {
      if (t >= len) continue;
      float* y = a.D + ((row0 + t) * H + head) * dv + col0;
#pragma unroll
      for (int c = 0; c < 8; ++c) {
        const int col = (c >> 2) * 64 + 4 * tx + (c & 3);
        if (col < nc) y[col] = acc[m][c];
      }
    }
  }
}

}  // namespace
}  // namespace prl

using namespace prl;
typedef __nv_bfloat16 bf16;

static bool geometry_ok(int heads, int kh, int dk, int dv, int taps) {
  return heads >= 1 && heads <= 65535 && kh >= 1 && heads % kh == 0 && dk >= 1 && dk <= 256 && dv >= 1 && dv <= 4096 && taps >= 1 && taps <= 16;
}

// fits: the CTA's vectors (unit q and k, its value heads' values and read-outs) in 200 KB of shared memory
extern "C" int32_t prl_gated_delta_step_fits(int32_t heads, int32_t kh, int32_t dk, int32_t dv, int32_t taps) {
  return geometry_ok(heads, kh, dk, dv, taps) && (2 * 256 + (int64_t)(heads / kh + 2) * dv) * 4 <= 200 * 1024;
}

extern "C" int prl_gated_delta_step(const float* P, int64_t ldp, int32_t off, int32_t off_b, int32_t off_a, int32_t off_g,
                                    const float* conv_w, int32_t taps, const float* A_log, const float* dt_bias, float unit_eps,
                                    const float* gain, float eps, int32_t heads, int32_t kh, int32_t dk, int32_t dv,
                                    const int32_t* seg_start, const int32_t* seg_len, const int32_t* seg_slot, int32_t n_seg,
                                    float* conv_state, float* state, void* out, int32_t f32, prl_stream_t st) {
  PRL_CHECK_ARG(P && conv_w && A_log && dt_bias && gain && seg_start && seg_len && seg_slot && conv_state && state && out,
                "prl_gated_delta_step: NULL argument");
  PRL_CHECK_ARG(n_seg >= 1 && n_seg <= 65535 && prl_gated_delta_step_fits(heads, kh, dk, dv, taps),
                "prl_gated_delta_step: bad shape (heads=%d q/k heads=%d dk=%d dv=%d taps=%d)", heads, kh, dk, dv, taps);
  const StepArgs a{P, ldp, off, off_b, off_a, off_g, conv_w, taps, A_log, dt_bias, unit_eps, gain, eps, heads, kh, dk, dv,
                   seg_start, seg_len, seg_slot, conv_state, state, out};
  const int rep = heads / kh, groups = rep > 1 ? 2 : 1, R = dk <= 32 ? 1 : dk <= 64 ? 2 : dk <= 128 ? 4 : 8;
  const bool vec = dk % 4 == 0 && ((uintptr_t)state & 15) == 0;
  const size_t smem = ((size_t)2 * 32 * R + (size_t)(groups + rep) * dv) * sizeof(float);
  static SmemAttr attr[16] = {};
#define PRL_GS(T, RR, VV, I)                                                                                                     \
  do {                                                                                                                           \
    if (smem > 48 * 1024) PRL_CUDA(ensure_smem((gated_delta_step_kernel<T, RR, VV>), (int)smem, attr[I]));                       \
    PRL_CUDA(launch_pdl((gated_delta_step_kernel<T, RR, VV>), dim3(kh, n_seg), dim3(256 * groups), smem, (cudaStream_t)st, a));  \
  } while (0)
#define PRL_GS2(RR, I)                                                                         \
  do {                                                                                         \
    if (f32) { if (vec) PRL_GS(float, RR, true, I); else PRL_GS(float, RR, false, I + 1); }    \
    else { if (vec) PRL_GS(bf16, RR, true, I + 2); else PRL_GS(bf16, RR, false, I + 3); }      \
  } while (0)
  if (R == 1) PRL_GS2(1, 0);
  else if (R == 2) PRL_GS2(2, 4);
  else if (R == 4) PRL_GS2(4, 8);
  else PRL_GS2(8, 12);
#undef PRL_GS2
#undef PRL_GS
  PRL_LAUNCH_CHECK();
  return PRL_OK;
}

// floats per row of the scratch of prl_gated_delta_split: W | E | gates
extern "C" int64_t prl_gated_delta_split_floats(int32_t heads, int32_t dk) { return (int64_t)heads * (dk + kPieceMax + 2); }

// Returns with y in `out` when dv <= 128; otherwise the raw read-out is in `D` and the head norm and gate are the caller's.
extern "C" int prl_gated_delta_split(const float* P, int64_t ldp, int32_t off, int32_t off_b, int32_t off_a, int32_t off_g,
                                     const float* conv_w, int32_t taps, const float* A_log, const float* dt_bias, float unit_eps,
                                     const float* gain, float eps, int32_t heads, int32_t kh, int32_t dk, int32_t dv, int32_t n_rows,
                                     const int32_t* row_slot, const int32_t* row_back, const int32_t* seg_start,
                                     const int32_t* seg_len, const int32_t* seg_slot, int32_t n_seg, const int32_t* seg_sub0,
                                     const int32_t* seg_nsub, const int32_t* sub_start, const int32_t* sub_len, int32_t n_sub,
                                     float* C, float* scratch, float* S0, float* D, float* conv_state, float* state, void* out,
                                     int32_t f32, prl_stream_t st_) {
  PRL_CHECK_ARG(P && conv_w && A_log && dt_bias && gain && row_slot && row_back && seg_start && seg_len && seg_slot && seg_sub0 &&
                seg_nsub && sub_start && sub_len && C && scratch && S0 && D && conv_state && state && out,
                "prl_gated_delta_split: NULL argument");
  PRL_CHECK_ARG(n_rows >= 1 && n_seg >= 1 && n_seg <= 65535 && n_sub >= 1 && geometry_ok(heads, kh, dk, dv, taps),
                "prl_gated_delta_split: bad shape (heads=%d q/k heads=%d dk=%d dv=%d taps=%d)", heads, kh, dk, dv, taps);
  SplitArgs a{P, ldp, off, off_b, off_a, off_g, conv_w, taps, A_log, dt_bias, unit_eps, gain, eps, heads, kh, dk, dv, 0,
              row_slot, row_back, seg_start, seg_len, seg_slot, seg_sub0, seg_nsub, sub_start, sub_len, C, nullptr, nullptr, nullptr, D,
              S0, conv_state, state, out};
  a.E = scratch;                                  // the widest first: 16-byte aligned rows whatever dk is
  a.W = scratch + (int64_t)n_rows * heads * kPieceMax;
  a.gates = a.W + (int64_t)n_rows * heads * dk;
  PRL_CHECK_ARG(((uintptr_t)scratch & 15) == 0, "prl_gated_delta_split: the scratch must be 16-byte aligned");
  a.vec = dk % 4 == 0 && dv % 4 == 0 && (((uintptr_t)C | (uintptr_t)S0 | (uintptr_t)D) & 15) == 0;
  cudaStream_t s = (cudaStream_t)st_;
  const bool tiled = a.vec && taps >= 2 && taps <= 4 && off % 4 == 0 && ldp % 4 == 0 && ((uintptr_t)P & 15) == 0;
  const dim3 gf((n_rows + kFrontRows - 1) / kFrontRows, (2 * kh + heads + kThreads / 32 - 1) / (kThreads / 32));
  if (tiled && taps == 2) PRL_CUDA(launch_pdl(gated_delta_front_tile_kernel<2>, gf, dim3(kThreads), (size_t)0, s, a, n_rows));
  else if (tiled && taps == 3) PRL_CUDA(launch_pdl(gated_delta_front_tile_kernel<3>, gf, dim3(kThreads), (size_t)0, s, a, n_rows));
  else if (tiled) PRL_CUDA(launch_pdl(gated_delta_front_tile_kernel<4>, gf, dim3(kThreads), (size_t)0, s, a, n_rows));
  else PRL_CUDA(launch_pdl(gated_delta_front_kernel, dim3(n_rows), dim3(kThreads), (size_t)0, s, a));
  PRL_LAUNCH_CHECK();
  const int dk4 = (dk + 3) & ~3, ldk = dk4 + 4;
  const size_t x_rows = (size_t)(kPieceMax - kBlk) * 2 * kPieceThreads, q_rows = (size_t)kPieceMax * ldk;
  const size_t sm_piece = (10 * (size_t)kBlkFloats + q_rows + (q_rows > x_rows ? q_rows : x_rows)) * sizeof(float);
  static SmemAttr at_piece = {};
  PRL_CUDA(ensure_smem(gated_delta_piece_kernel, (int)sm_piece, at_piece));
  PRL_CUDA(launch_pdl(gated_delta_piece_kernel, dim3(n_sub, heads), dim3(kPieceThreads), sm_piece, s, a));
  PRL_LAUNCH_CHECK();
  const dim3 gw((dv + kWalkCols - 1) / kWalkCols, heads, n_seg);
  // partial sums: four quarters of the key channels for 64 rows, later one half of the update
  const size_t red = (size_t)kWalkCols * (4 * kPieceMax > dk4 ? 4 * kPieceMax : dk4);
  const int stages = dk4 <= 128 && (int64_t)gw.x * gw.y * gw.z <= num_sms() ? 2 : 1;
  const size_t sm_walk = ((size_t)stages * 2 * kPieceMax * ldk + (size_t)(dk4 + kPieceMax) * (kWalkCols + 4) + red) * sizeof(float);
  static SmemAttr at_walk[2] = {};
  if (stages == 2) {
    PRL_CUDA(ensure_smem(gated_delta_walk_kernel<2>, (int)sm_walk, at_walk[0]));
    PRL_CUDA(launch_pdl(gated_delta_walk_kernel<2>, gw, dim3(kThreads), sm_walk, s, a));
  } else {
    PRL_CUDA(ensure_smem(gated_delta_walk_kernel<1>, (int)sm_walk, at_walk[1]));
    PRL_CUDA(launch_pdl(gated_delta_walk_kernel<1>, gw, dim3(kThreads), sm_walk, s, a));
  }
  PRL_LAUNCH_CHECK();
  const size_t sm_read = (size_t)2 * (kPieceMax * 36 + 32 * (kOutCols + 4)) * sizeof(float);
  const dim3 gr(n_sub, heads, (dv + kOutCols - 1) / kOutCols);
  static SmemAttr at_read[3] = {};
#define PRL_GR(T, NORM, I)                                                                                   \
  do {                                                                                                       \
    PRL_CUDA(ensure_smem((gated_delta_read_kernel<T, NORM>), (int)sm_read, at_read[I]));                     \
    PRL_CUDA(launch_pdl((gated_delta_read_kernel<T, NORM>), gr, dim3(kThreads), sm_read, s, a));             \
  } while (0)
  if (dv > kOutCols) PRL_GR(float, false, 0);
  else if (f32) PRL_GR(float, true, 1);
  else PRL_GR(bf16, true, 2);
#undef PRL_GR
  PRL_LAUNCH_CHECK();
  return PRL_OK;
}
