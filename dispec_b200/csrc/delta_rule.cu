// The gated delta rule as a recurrence over a matrix state, in 32-bit floats on the FMA units:
//
//     S <- g_t S;   u_t = beta_t (v_t - S^T k_t);   S <- S + k_t u_t^T;   o_t = S^T q_t
//
// (S: [dim, vdim] per head and request, zero at admission, in the request's state slot between steps, so
// that a prompt can be cut into portions anywhere and decoded tokens continue from what it left.)  Rows
// are floats: q and k for each of G groups of heads, v for each of H heads, head h reading q and k of group
// h / (H / G); `steps` [T, 2, H] holds beta and ln g of every token and head.
//
// Single tokens (delta_single_kernel): a block takes 32 value columns of one head and request, reads its part
// of the state once into registers, forms S^T k and S^T q of the old state together,
//     u = beta (v - g S^T k),   o = g S^T q + (k . q) u,   S <- g S + k u^T,
// and writes it back.  Portions run through it too where the state has more than 256 rows.
//
// Portions of prompts, eight tokens at a time.  With gamma_i = g_1 .. g_i and D_ij = gamma_i / gamma_j within a
// run of eight and S0 the state in front of it, the u_i solve a unit lower triangular system,
//     u_i = beta_i (v_i - gamma_i S0^T k_i - sum_{j<i} D_ij (k_i . k_j) u_j)
//     o_i = gamma_i S0^T q_i + sum_{j<=i} D_ij (k_j . q_i) u_j
//     S   = gamma_8 S0 + sum_j D_8j k_j u_j^T
// so that with x_j = v_j - gamma_j S0^T k_j both are fixed 8 x 8 matrices times x: u = P x, o = gamma S0^T q + N x.
//   delta_prepare_kernel   forms P (rows already times D_8i) and N of every run and head, all runs in parallel
//                          (`coef` [T, H, 20]: row i of P, row i of N, gamma_i, gamma_8, two spare).
//   delta_runs_kernel      the sequential part: a block takes 8 value columns of one head and request and walks
//                          its runs; the state stays in registers (a warp holds 32 state rows, eight lanes
//                          share the rows of a column), the products S0^T k and S0^T q of eight tokens are added
//                          over lanes together (each exchange halves what a lane still holds; a lane counts the tokens
//                          from its own, so that what it keeps always comes first) and over warps in shared memory; rows arrive by cp.async two runs ahead.
// A request whose first row carries a negative position (a padding row of a captured step) is skipped: its
// state slot belongs to someone else.
#include "common.cuh"

namespace {

constexpr int RUN = 8, COEF = 20, SLICES = 8, COLS = 8;

struct DeltaArgs {
  const float* rows;  // [T, ld]
  long ld;
  int q_off, k_off, v_off;
  const float* steps;  // [T, 2, H]: beta, ln g
  int H, G, dim, vdim;
  float* state;  // [slots, H, dim, vdim]
  const int* state_slot;
  const int* q_start;
  const int* positions;
  float* out;  // [T, ldo]
  long ldo;
  float* coef;  // [T, H, COEF]
  int first_seq;
};

// ------------------------------------------------------------------------------- single tokens
// 128 threads: thread = (8 groups of four columns) x (16 groups of state rows), ROWS rows a thread
template <int ROWS>
__global__ void __launch_bounds__(128) delta_single_kernel(const DeltaArgs p) {
  extern __shared__ __align__(16) float smem[];
  float* ks = smem;                    // [dim]
  float* qs = smem + p.dim;            // [dim]
  __shared__ __align__(16) float4 part[4][8][2];
  const int seq = p.first_seq + blockIdx.z, head = blockIdx.y, group = head / (p.H / p.G);
  const int t0 = p.q_start[seq], t1 = p.q_start[seq + 1];
  if (t1 <= t0 || p.positions[t0] < 0) return;
  const int tid = threadIdx.x, tx = tid & 7, ty = tid >> 3, lane = tid & 31, warp = tid >> 5;
  const int col = blockIdx.x * 32 + tx * 4;
  const bool wide = p.vdim % 4 == 0;
  float* sp = p.state + ((size_t)p.state_slot[seq] * p.H + head) * p.dim * p.vdim;
  float4 S[ROWS];
#pragma unroll
  for (int i = 0; i < ROWS; ++i) {
    const int r = ty + 16 * i;
    S[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (r >= p.dim || col >= p.vdim) continue;
    const float* src = sp + (size_t)r * p.vdim + col;
    if (wide) {
      S[i] = *reinterpret_cast<const float4*>(src);
    } else {
      S[i].x = src[0];
      if (col + 1 < p.vdim) S[i].y = src[1];
      if (col + 2 < p.vdim) S[i].z = src[2];
      if (col + 3 < p.vdim) S[i].w = src[3];
    }
  }
  for (int t = t0; t < t1; ++t) {
    const float* row = p.rows + (size_t)t * p.ld;
    if (t > t0) __syncthreads();  // the rows are taken again
    for (int i = tid; i < p.dim; i += 128) {
      ks[i] = row[p.k_off + (size_t)group * p.dim + i];
      qs[i] = row[p.q_off + (size_t)group * p.dim + i];
    }
    const float beta = p.steps[(size_t)t * 2 * p.H + head], g = expf(p.steps[((size_t)t * 2 + 1) * p.H + head]);
    float v[4];
#pragma unroll
    for (int c = 0; c < 4; ++c) v[c] = col + c < p.vdim ? row[p.v_off + (size_t)head * p.vdim + col + c] : 0.f;
    __syncthreads();
    float kq = 0.f;
    for (int i = lane; i < p.dim; i += 32) kq = fmaf(ks[i], qs[i], kq);
    kq = warp_sum(kq);
    float a[8] = {};  // S^T k, S^T q of this thread's columns
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
      const int r = ty + 16 * i;
      if (r >= p.dim) continue;
      const float kv = ks[r], qv = qs[r];
      a[0] = fmaf(S[i].x, kv, a[0]);
      a[1] = fmaf(S[i].y, kv, a[1]);
      a[2] = fmaf(S[i].z, kv, a[2]);
      a[3] = fmaf(S[i].w, kv, a[3]);
      a[4] = fmaf(S[i].x, qv, a[4]);
      a[5] = fmaf(S[i].y, qv, a[5]);
      a[6] = fmaf(S[i].z, qv, a[6]);
      a[7] = fmaf(S[i].w, qv, a[7]);
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      a[e] += __shfl_xor_sync(0xffffffffu, a[e], 8);
      a[e] += __shfl_xor_sync(0xffffffffu, a[e], 16);
    }
    if (lane < 8) {
      part[warp][tx][0] = make_float4(a[0], a[1], a[2], a[3]);
      part[warp][tx][1] = make_float4(a[4], a[5], a[6], a[7]);
    }
    __syncthreads();
    float4 r4 = part[0][tx][0], o4 = part[0][tx][1];
#pragma unroll
    for (int w = 1; w < 4; ++w) {
      const float4 r = part[w][tx][0], o = part[w][tx][1];
      r4.x += r.x, r4.y += r.y, r4.z += r.z, r4.w += r.w;
      o4.x += o.x, o4.y += o.y, o4.z += o.z, o4.w += o.w;
    }
    const float u[4] = {beta * (v[0] - g * r4.x), beta * (v[1] - g * r4.y), beta * (v[2] - g * r4.z), beta * (v[3] - g * r4.w)};
    if (ty == 0) {
      const float o[4] = {fmaf(kq, u[0], g * o4.x), fmaf(kq, u[1], g * o4.y), fmaf(kq, u[2], g * o4.z), fmaf(kq, u[3], g * o4.w)};
      float* dst = p.out + (size_t)t * p.ldo + (size_t)head * p.vdim + col;
#pragma unroll
      for (int c = 0; c < 4; ++c)
        if (col + c < p.vdim) dst[c] = o[c];
    }
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
      const int r = ty + 16 * i;
      const float kv = r < p.dim ? ks[r] : 0.f;
      S[i].x = fmaf(g, S[i].x, kv * u[0]);
      S[i].y = fmaf(g, S[i].y, kv * u[1]);
      S[i].z = fmaf(g, S[i].z, kv * u[2]);
      S[i].w = fmaf(g, S[i].w, kv * u[3]);
    }
  }
#pragma unroll
  for (int i = 0; i < ROWS; ++i) {
    const int r = ty + 16 * i;
    if (r >= p.dim || col >= p.vdim) continue;
    float* dst = sp + (size_t)r * p.vdim + col;
    if (wide) {
      *reinterpret_cast<float4*>(dst) = S[i];
    } else {
      dst[0] = S[i].x;
      if (col + 1 < p.vdim) dst[1] = S[i].y;
      if (col + 2 < p.vdim) dst[2] = S[i].z;
      if (col + 3 < p.vdim) dst[3] = S[i].w;
    }
  }
}

// ------------------------------------------------------------------------------- portions: coefficients
// A block of 64 threads takes one run of up to eight tokens and one group of heads.  run_seq / run_tok0: the
// step's list of runs (their request and first token).
__global__ void __launch_bounds__(64)
delta_prepare_kernel(const DeltaArgs p, const int* __restrict__ run_seq, const int* __restrict__ run_tok0, int run_offset) {
  extern __shared__ __align__(16) float smem[];
  __shared__ float kk[RUN][RUN + 1], qk[RUN][RUN + 1];  // [i][j]: k_i . k_j and q_i . k_j
  __shared__ float tri[2][RUN][RUN + 1], mix[2][RUN][RUN + 1];
  const int run = run_offset + blockIdx.x, group = blockIdx.y;
  const int seq = run_seq[run], tok0 = run_tok0[run];
  const int row0 = p.q_start[seq] + tok0, n = min(RUN, p.q_start[seq + 1] - row0);
  if (n <= 0 || p.positions[row0] < 0) return;
  const int tid = threadIdx.x, ldm = (p.dim + 3) / 4 * 4 + 4;
  float* ks = smem;             // [RUN][ldm]
  float* qs = smem + RUN * ldm;
  const bool wide = p.dim % 4 == 0 && p.ld % 4 == 0 && p.k_off % 4 == 0 && p.q_off % 4 == 0 && ((uintptr_t)p.rows & 15) == 0;
#pragma unroll
  for (int r = 0; r < RUN; ++r) {
    const float* row = p.rows + (size_t)(row0 + min(r, n - 1)) * p.ld + (size_t)group * p.dim;
    if (wide) {
      for (int i = tid * 4; i < p.dim; i += 256) {
        *reinterpret_cast<float4*>(ks + r * ldm + i) = r < n ? *reinterpret_cast<const float4*>(row + p.k_off + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        *reinterpret_cast<float4*>(qs + r * ldm + i) = r < n ? *reinterpret_cast<const float4*>(row + p.q_off + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      }
    } else {
      for (int i = tid; i < ldm; i += 64) {
        ks[r * ldm + i] = r < n && i < p.dim ? row[p.k_off + i] : 0.f;
        qs[r * ldm + i] = r < n && i < p.dim ? row[p.q_off + i] : 0.f;
      }
    }
  }
  __syncthreads();
  {
    const int i = tid >> 3, j = tid & 7;
    float a[4] = {}, b[4] = {};
    for (int d = 0; d < ldm - 4; d += 4) {
      const float4 kj = *reinterpret_cast<const float4*>(ks + j * ldm + d), ki = *reinterpret_cast<const float4*>(ks + i * ldm + d);
      const float4 qi = *reinterpret_cast<const float4*>(qs + i * ldm + d);
      a[0] = fmaf(ki.x, kj.x, a[0]);
      a[1] = fmaf(ki.y, kj.y, a[1]);
      a[2] = fmaf(ki.z, kj.z, a[2]);
      a[3] = fmaf(ki.w, kj.w, a[3]);
      b[0] = fmaf(qi.x, kj.x, b[0]);
      b[1] = fmaf(qi.y, kj.y, b[1]);
      b[2] = fmaf(qi.z, kj.z, b[2]);
      b[3] = fmaf(qi.w, kj.w, b[3]);
    }
    kk[i][j] = (a[0] + a[1]) + (a[2] + a[3]);
    qk[i][j] = (b[0] + b[1]) + (b[2] + b[3]);
  }
  __syncthreads();
  // a warp a head: lane = column c of the matrices (lanes 0 .. 7)
  const int warp = tid >> 5, lane = tid & 31, c = lane & 7, per = p.H / p.G;
  for (int a = warp; a < per; a += 2) {
    const int head = group * per + a;
    const size_t st = (size_t)(row0 + min(c, n - 1)) * 2 * p.H + head;
    const float beta = c < n ? p.steps[st] : 0.f, lg = c < n ? p.steps[st + p.H] : 0.f;
    float L = lg;  // ln gamma_c
#pragma unroll
    for (int o = 1; o < RUN; o <<= 1) {
      const float y = __shfl_up_sync(0xffffffffu, L, o, RUN);
      if (c >= o) L += y;
    }
    const float Lend = __shfl_sync(0xffffffffu, L, RUN - 1, RUN);
    float (*A)[RUN + 1] = tri[warp], (*M)[RUN + 1] = mix[warp];
    __syncwarp();
#pragma unroll
    for (int i = 0; i < RUN; ++i) {
      const float Li = __shfl_sync(0xffffffffu, L, i, RUN), bi = __shfl_sync(0xffffffffu, beta, i, RUN);
      if (lane < RUN) {
        const float D = c <= i ? expf(Li - L) : 0.f;
        A[i][c] = c < i ? bi * D * kk[i][c] : 0.f;
        M[i][c] = D * qk[i][c];
      }
    }
    __syncwarp();
    float x[RUN];  // column c of the inverse of (I + A), times beta_c
#pragma unroll
    for (int i = 0; i < RUN; ++i) {
      float s = i == c ? beta : 0.f;
#pragma unroll
      for (int j = 0; j < RUN; ++j)
        if (j < i) s = fmaf(-A[i][j], x[j], s);
      x[i] = s;
    }
#pragma unroll
    for (int i = 0; i < RUN; ++i) {
      float s = 0.f;
#pragma unroll
      for (int j = 0; j < RUN; ++j)
        if (j <= i) s = fmaf(M[i][j], x[j], s);
      const float Li = __shfl_sync(0xffffffffu, L, i, RUN);
      if (i < n && lane < RUN) {
        float* dst = p.coef + ((size_t)(row0 + i) * p.H + head) * COEF;
        dst[c] = expf(Lend - Li) * x[i];
        dst[RUN + c] = s;
        if (c == 0) dst[2 * RUN] = expf(Li);
        if (c == 1) dst[2 * RUN + 1] = expf(Lend);
        if (c == 2 || c == 3) dst[2 * RUN + c] = 0.f;
      }
    }
  }
}

// ------------------------------------------------------------------------------- portions: the walk
typedef unsigned long long f32x2;  // two 32-bit floats side by side: one instruction, each half rounded as its scalar form is
__device__ __forceinline__ f32x2 pack2f(float a, float b) {
  f32x2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ void unpack2f(f32x2 v, float& a, float& b) { asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v)); }
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
  f32x2 r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ void cp_async4(float* smem, const float* gmem) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"((uint32_t)__cvta_generic_to_shared(smem)), "l"(gmem));
}
__device__ __forceinline__ void cp_async16(float* smem, const float* gmem) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((uint32_t)__cvta_generic_to_shared(smem)), "l"(gmem));
}

template <int PARTS>
struct Walk {
  static constexpr int rows = 32 * PARTS;                                        // state rows, padded
  static constexpr int stage = RUN * (2 * rows + COLS + COEF);                   // k, q, v, coefficients of a run
  static constexpr int stages = 4;
  static constexpr int token = 2 * COLS + 4;                                     // a token's S^T k and S^T q of the block's columns
  static constexpr int meet = PARTS * RUN * token;
  static constexpr size_t smem = sizeof(float) * (stages * stage + meet + RUN * COLS);
};

// PARTS warps of 32 state rows; SLICES lanes share the rows of a column, a lane holds 32 / SLICES rows of two columns
template <int PARTS>
__global__ void __launch_bounds__(32 * PARTS) delta_runs_kernel(const DeltaArgs p) {
  using L = Walk<PARTS>;
  constexpr int ROWS = 32 / SLICES, NC = 2, THREADS = 32 * PARTS, DP = L::rows;
  static_assert(RUN == SLICES && COLS == NC * 32 / SLICES, "a lane ends with one token, a warp covers the block's columns");
  extern __shared__ __align__(16) float smem[];
  float* meet = smem + L::stages * L::stage;
  float* us = meet + L::meet;  // [RUN][COLS]
  const int seq = p.first_seq + blockIdx.z, head = blockIdx.y, group = head / (p.H / p.G);
  const int t0 = p.q_start[seq], t1 = p.q_start[seq + 1];
  if (t1 <= t0 || p.positions[t0] < 0) return;
  const int tid = threadIdx.x, lane = tid & 31, part = tid >> 5;
  // neighbouring lanes share rows (loads of 16 bytes at one address by neighbours cost half of what they cost spread
  // over the warp), cl: this lane's first column within the block's
  constexpr int GROUPS = 32 / SLICES;
  const int slice = lane / GROUPS, cl = lane % GROUPS * NC;
  const int row0 = part * 32 + slice * ROWS, col0 = blockIdx.x * COLS;
  float* sp = p.state + ((size_t)p.state_slot[seq] * p.H + head) * p.dim * p.vdim;

  f32x2 S[ROWS / 2][NC];
#pragma unroll
  for (int k = 0; k < ROWS / 2; ++k)
#pragma unroll
    for (int c = 0; c < NC; ++c) {
      const int r = row0 + 2 * k, cc = col0 + cl + c;
      const float a = r < p.dim && cc < p.vdim ? sp[(size_t)r * p.vdim + cc] : 0.f;
      const float b = r + 1 < p.dim && cc < p.vdim ? sp[(size_t)(r + 1) * p.vdim + cc] : 0.f;
      S[k][c] = pack2f(a, b);
    }
  const bool aligned = p.ld % 4 == 0 && ((uintptr_t)p.rows & 15) == 0;
  const bool wide = aligned && p.dim % 4 == 0 && p.q_off % 4 == 0 && p.k_off % 4 == 0;
  const bool v_wide = aligned && p.vdim % 4 == 0 && p.v_off % 4 == 0;

  // what no copy fills (rows beyond dim, columns beyond vdim) is zero in every stage from here on
  for (int i = tid; i < L::stages * L::stage; i += THREADS) smem[i] = 0.f;
  __syncthreads();

  // this thread's pieces of a run: where the first two lie in the rows, and the coefficients'
  const int piece_r = tid / (DP / 4), piece_i = tid % (DP / 4) * 4;
  const bool piece_on = wide && piece_i < p.dim;
  const float* row_piece = p.rows + (size_t)piece_r * p.ld + (size_t)group * p.dim + piece_i;
  const int val_r = tid / (COLS / 4), val_i = tid % (COLS / 4) * 4;
  const bool val_on = v_wide && tid < RUN * COLS / 4 && col0 + val_i < p.vdim;
  const float* val_piece = p.rows + (size_t)val_r * p.ld + p.v_off + (size_t)head * p.vdim + col0 + val_i;
  auto stage_run = [&](int base, float* buf) {
    const int n = min(RUN, t1 - base);
    if (n < RUN) {  // the last run: its missing tokens are rows of zeros
      for (int i = tid; i < (RUN - n) * DP; i += THREADS) {
        buf[n * DP + i] = 0.f;
        buf[(RUN + n) * DP + i] = 0.f;
      }
      for (int i = tid; i < (RUN - n) * COLS; i += THREADS) buf[2 * RUN * DP + n * COLS + i] = 0.f;
      for (int i = tid; i < (RUN - n) * COEF; i += THREADS) buf[2 * RUN * DP + RUN * COLS + n * COEF + i] = 0.f;
    }
    static_assert(RUN * DP / 4 == 2 * THREADS, "two 16-byte pieces a thread and plane");
#pragma unroll
    for (int pl = 0; pl < 2; ++pl) {
      float* dst = buf + pl * RUN * DP;
      if (wide) {
        const float* src = row_piece + (size_t)base * p.ld + (pl == 0 ? p.k_off : p.q_off);
        if (piece_on && piece_r < n) cp_async16(dst + piece_r * DP + piece_i, src);
        if (piece_on && piece_r + RUN / 2 < n) cp_async16(dst + (piece_r + RUN / 2) * DP + piece_i, src + RUN / 2 * p.ld);
      } else {
        const float* src = p.rows + (size_t)base * p.ld + (pl == 0 ? p.k_off : p.q_off) + (size_t)group * p.dim;
        for (int idx = tid; idx < n * DP; idx += THREADS) {
          const int r = idx / DP, i = idx % DP;
          if (i < p.dim) cp_async4(dst + r * DP + i, src + (size_t)r * p.ld + i);
        }
      }
    }
    float* vs = buf + 2 * RUN * DP;
    if (v_wide) {
      if (val_on && val_r < n) cp_async16(vs + val_r * COLS + val_i, val_piece + (size_t)base * p.ld);
    } else {
      const float* vsrc = p.rows + (size_t)base * p.ld + p.v_off + (size_t)head * p.vdim + col0;
      for (int idx = tid; idx < n * COLS; idx += THREADS) {
        const int r = idx / COLS, i = idx % COLS;
        if (col0 + i < p.vdim) cp_async4(vs + idx, vsrc + (size_t)r * p.ld + i);
      }
    }
    float* cs = vs + RUN * COLS;
#pragma unroll
    for (int idx = THREADS - 1 - tid; idx < RUN * (COEF / 4); idx += THREADS)  // (from the other end: the first threads have the values)
      if (idx < n * (COEF / 4)) cp_async16(cs + idx * 4, p.coef + ((size_t)(base + idx / (COEF / 4)) * p.H + head) * COEF + idx % (COEF / 4) * 4);
  };

#pragma unroll
  for (int s = 0; s < 2; ++s) {
    if (t0 + s * RUN < t1) stage_run(t0 + s * RUN, smem + s * L::stage);
    asm volatile("cp.async.commit_group;\n");
  }
  asm volatile("cp.async.wait_group 1;\n");
  __syncthreads();

  int mine[RUN];  // where this lane's rows of token t ^ slice lie in a stage
#pragma unroll
  for (int t = 0; t < RUN; ++t) mine[t] = (t ^ slice) * DP + row0;

  int turn = 0;
  for (int base = t0; base < t1; base += RUN, turn = (turn + 1) & 3) {
    const float* buf = smem + turn * L::stage;
    // two runs ahead, into the stage of two runs ago (everyone has passed a barrier since it was last read)
    if (base + 2 * RUN < t1) stage_run(base + 2 * RUN, smem + ((turn + 2) & 3) * L::stage);
    asm volatile("cp.async.commit_group;\n");

    // S0^T k and S0^T q of the run's tokens over this lane's rows; t counts from this lane's token: value
    // (t * 2 + which) * NC + column belongs to token t ^ slice
    static_assert(ROWS == 4, "a lane's rows are one 16-byte piece");
    float acc[RUN * 2 * NC];
    ulonglong2 kr[RUN], qr[RUN];  // the keys stay for the update of the state
#pragma unroll
    for (int t = 0; t < RUN; ++t) {
      kr[t] = *reinterpret_cast<const ulonglong2*>(buf + mine[t]);
      qr[t] = *reinterpret_cast<const ulonglong2*>(buf + RUN * DP + mine[t]);
    }
#pragma unroll
    for (int t = 0; t < RUN; ++t)
#pragma unroll
      for (int w = 0; w < 2; ++w) {
        const ulonglong2 x = w == 0 ? kr[t] : qr[t];
        f32x2 s[NC];
#pragma unroll
        for (int c = 0; c < NC; ++c) s[c] = fma2(S[1][c], x.y, mul2(S[0][c], x.x));
#pragma unroll
        for (int c = 0; c < NC; ++c) {
          float a, b;
          unpack2f(s[c], a, b);
          acc[(t * 2 + w) * NC + c] = a + b;
        }
      }
    // sums over the slices: each exchange leaves a lane the first half of its values (the tokens nearer to its own, whose
    // partner's are in that partner's second half), at the end those of token `slice`
#pragma unroll
    for (int o = SLICES / 2, m = RUN * NC; o > 0; o >>= 1, m >>= 1) {
#pragma unroll
      for (int i = 0; i < RUN * NC; ++i)
        if (i < m) acc[i] += __shfl_xor_sync(0xffffffffu, acc[i + m], o * GROUPS);
    }
    {
      float* dst = meet + (part * RUN + slice) * L::token + cl;
      *reinterpret_cast<float2*>(dst) = make_float2(acc[0], acc[1]);
      *reinterpret_cast<float2*>(dst + COLS) = make_float2(acc[2], acc[3]);
    }
    __syncthreads();
    // u and o: a thread a (token, column), the eight tokens of a column in neighbouring lanes
    const float* vs = buf + 2 * RUN * DP;
    const float* cs = vs + RUN * COLS;
#pragma unroll
    for (int idx = tid; idx < RUN * COLS; idx += THREADS) {
      const int t = idx & 7, c = idx >> 3;
      float r = 0.f, o = 0.f;
#pragma unroll
      for (int w = 0; w < PARTS; ++w) {
        const float* m = meet + (w * RUN + t) * L::token + c;
        r += m[0];
        o += m[COLS];
      }
      const float* cf = cs + t * COEF;
      float P[RUN], N[RUN];
#pragma unroll
      for (int j = 0; j < RUN; j += 4) {
        *reinterpret_cast<float4*>(P + j) = *reinterpret_cast<const float4*>(cf + j);
        *reinterpret_cast<float4*>(N + j) = *reinterpret_cast<const float4*>(cf + RUN + j);
      }
      const float gamma = cf[2 * RUN], x = vs[t * COLS + c] - gamma * r;
      o *= gamma;
      float u = 0.f, u2 = 0.f, o2 = 0.f;
#pragma unroll
      for (int j = 0; j < RUN; j += 2) {
        const float xj = __shfl_sync(0xffffffffu, x, j, RUN), xk = __shfl_sync(0xffffffffu, x, j + 1, RUN);
        u = fmaf(P[j], xj, u);
        o = fmaf(N[j], xj, o);
        u2 = fmaf(P[j + 1], xk, u2);
        o2 = fmaf(N[j + 1], xk, o2);
      }
      u += u2;
      o += o2;
      us[t * COLS + c] = u;
      if (base + t < t1 && col0 + c < p.vdim) p.out[(size_t)(base + t) * p.ldo + (size_t)head * p.vdim + col0 + c] = o;
    }
    asm volatile("cp.async.wait_group 1;\n");
    __syncthreads();  // the u are there; so is the next run's stage
    const float g = cs[2 * RUN + 1];
    const f32x2 g2 = pack2f(g, g);
#pragma unroll
    for (int k = 0; k < ROWS / 2; ++k)
#pragma unroll
      for (int c = 0; c < NC; ++c) S[k][c] = mul2(g2, S[k][c]);
    float2 u[RUN];  // both columns of token t ^ slice
#pragma unroll
    for (int t = 0; t < RUN; ++t) u[t] = *reinterpret_cast<const float2*>(us + (t ^ slice) * COLS + cl);
#pragma unroll
    for (int t = 0; t < RUN; ++t) {
      const f32x2 ua = pack2f(u[t].x, u[t].x), ub = pack2f(u[t].y, u[t].y);
      S[0][0] = fma2(kr[t].x, ua, S[0][0]);
      S[0][1] = fma2(kr[t].x, ub, S[0][1]);
      S[1][0] = fma2(kr[t].y, ua, S[1][0]);
      S[1][1] = fma2(kr[t].y, ub, S[1][1]);
    }
  }
  asm volatile("cp.async.wait_group 0;\n");
#pragma unroll
  for (int k = 0; k < ROWS / 2; ++k)
#pragma unroll
    for (int c = 0; c < NC; ++c) {
      const int r = row0 + 2 * k, cc = col0 + cl + c;
      float a, b;
      unpack2f(S[k][c], a, b);
      if (r < p.dim && cc < p.vdim) sp[(size_t)r * p.vdim + cc] = a;
      if (r + 1 < p.dim && cc < p.vdim) sp[(size_t)(r + 1) * p.vdim + cc] = b;
    }
}

template <int ROWS>
int launch_single(const DeltaArgs& a, int S, cudaStream_t stream) {
  const dim3 grid((a.vdim + 31) / 32, a.H, S);
  DSP_CUDA(launch_plain(delta_single_kernel<ROWS>, grid, dim3(128), 2 * (size_t)a.dim * sizeof(float), stream, a));
  DSP_CHECK_LAUNCH("dsp_delta_rule");
  return 0;
}

template <int PARTS>
int launch_runs(const DeltaArgs& a, int S, cudaStream_t stream) {
  static bool configured = false;
  if (!configured) {
    DSP_CUDA(cudaFuncSetAttribute(delta_runs_kernel<PARTS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)Walk<PARTS>::smem));
    configured = true;
  }
  const dim3 grid((a.vdim + COLS - 1) / COLS, a.H, S);
  DSP_CUDA(launch_plain(delta_runs_kernel<PARTS>, grid, dim3(32 * PARTS), Walk<PARTS>::smem, stream, a));
  DSP_CHECK_LAUNCH("dsp_delta_rule");
  return 0;
}
}  // namespace

// The first `num_single` requests bring one token each; of the list of runs (eight tokens a run) theirs come
// first.  `coef` (float [T, H, 20], 16-byte aligned) is needed where a request brings more.
extern "C" int dsp_delta_rule(const float* rows, long ld, int q_off, int k_off, int v_off, const float* steps, int H, int G,
                              int dim, int vdim, float* state, const int* state_slot, const int* q_start, const int* positions,
                              const int* run_seq, const int* run_tok0, int num_runs, float* out, long ldo, int S,
                              int num_single, float* coef, cudaStream_t stream) {
  if (S == 0) return 0;
  DSP_REQUIRE(rows && steps && state && state_slot && q_start && positions && out, "dsp_delta_rule: missing operand");
  DSP_REQUIRE(H > 0 && G > 0 && H % G == 0 && H <= 65535 && S <= 65535, "dsp_delta_rule: H=%d, G=%d, S=%d", H, G, S);
  DSP_REQUIRE(dim > 0 && dim <= 512 && vdim > 0, "dsp_delta_rule: dim=%d (at most 512), vdim=%d", dim, vdim);
  DSP_REQUIRE(num_single >= 0 && num_single <= S, "dsp_delta_rule: %d single tokens of %d requests", num_single, S);
  DeltaArgs a = {rows, ld, q_off, k_off, v_off, steps, H, G, dim, vdim, state, state_slot, q_start, positions, out, ldo, coef, 0};
  const bool walk = dim <= 256;  // states with more rows take their portions token by token
  const int single = walk ? num_single : S;
  if (single > 0) {
    int rc;
    if (dim <= 32) rc = launch_single<2>(a, single, stream);
    else if (dim <= 64) rc = launch_single<4>(a, single, stream);
    else if (dim <= 128) rc = launch_single<8>(a, single, stream);
    else if (dim <= 256) rc = launch_single<16>(a, single, stream);
    else rc = launch_single<32>(a, single, stream);
    if (rc) return rc;
  }
  const int rest = S - single, runs = num_runs - single;
  if (rest <= 0) return 0;
  DSP_REQUIRE(coef && ((uintptr_t)coef & 15) == 0 && run_seq && run_tok0 && runs > 0, "dsp_delta_rule: portions without their runs or scratch");
  a.first_seq = single;
  DSP_CUDA(launch_plain(delta_prepare_kernel, dim3(runs, G), dim3(64), 2 * RUN * ((size_t)(dim + 3) / 4 * 4 + 4) * sizeof(float),
                        stream, a, run_seq, run_tok0, single));
  DSP_CHECK_LAUNCH("dsp_delta_rule (coefficients)");
  if (dim <= 32) return launch_runs<1>(a, rest, stream);
  if (dim <= 64) return launch_runs<2>(a, rest, stream);
  if (dim <= 128) return launch_runs<4>(a, rest, stream);
  return launch_runs<8>(a, rest, stream);
}
