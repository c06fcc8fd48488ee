// Linear attention as a recurrence over a matrix state, in 32-bit floats on the FMA units:
//
//     S_t = diag(a_t) S_(t-1) + b_t v_t^T        (S: [dim, vdim] per head and request)
//     o_t = S_t^T q_t
//
// The state of a request lives in its state slot between steps, so a prompt can be cut into
// portions anywhere and decoded tokens continue from what the prompt left.  What a_t, b_t and
// q_t are is the mixer's business; four forms are built in, all computed here from the raw
// rows of the mixer's fused projection (float or bfloat16), in 32-bit:
//
//   FIXED_DECAY   a_t = decay[head] (one number per head); q_t and b_t are the projected query
//                 and key with pairs (i, i + rot/2) of their first `rot` dimensions turned by
//                 the angle position * inv_freq[i], and b_t scaled by `key_scale` afterwards;
//                 with `act` = 1 the raw query, key and value pass through silu first
//   FORGET_GATE   a_t = f_t = lower + (1 - lower) * sigmoid(raw_f + bias), b_t = 1 - f_t,
//                 q_t = silu(raw_q)      (lower and bias per head and channel)
//   KEY_DECAY     q_t = raw_q * q_scale, b_t = raw_k * key_scale, a_t = sigmoid(z)^power with z = M r + bias
//                 per head and channel, r the `rank` columns of the row from `low_off` on and M given
//                 transposed ([rank, H * dim])
//   STEP_DECAY    rows of floats; q_t and b_t are columns shared by the heads of a group, a_t one number per
//                 token and head and the value scaled by another (`steps`); o_t gets skip[head] * v_t on top:
//                     S_t = a S_(t-1) + step b_t v_t^T,   o_t = S_t^T q_t + skip v_t
//
// One block per (request, head, tile of value columns); what a block computes is sequential in the
// tokens of its request.  A thread holds a tile of the state in registers, a few neighbouring rows of four
// neighbouring columns, so that what it reads of q, b and a serves four columns; rows go through the
// multipliers in pairs.  Eight tokens' partial outputs are added over the lanes that share columns together,
// each exchange halving the values a lane still holds.  Tokens are staged through shared memory in rounds.
// Portions of prompts: a first, fully parallel kernel writes q_t, b_t (and a_t) of every token as floats
// (STEP_DECAY streams its rows as they are), and the recurrence streams them in with cp.async, two rounds
// ahead of the one that is computed; eight lanes cover 16 (32) state rows and groups of warps the rest (a lone
// prompt leaves an SM one block: eight warps hide one another's latencies), the groups' results meet in
// shared memory and leave one round later.  Single tokens: transformed as they are staged, in one kernel,
// the lanes of a warp cover all the rows.
// State rows beyond 256 take a kernel of their own with one column a thread.  A request whose first row
// carries a negative position (a padding row of a captured step) is skipped: its state slot belongs to
// someone else.
#include <type_traits>

#include "common.cuh"

namespace {

enum { FIXED_DECAY = 0, FORGET_GATE = 1, KEY_DECAY = 2, STEP_DECAY = 3 };
enum { SCALAR_DECAY = 0, VECTOR_DECAY = 1, TOKEN_DECAY = 2 };  // what a_t is: kinds of the kernel
constexpr int THREADS = 256;

struct RecurrenceArgs {
  const void* proj;  // [T, ld]: raw projection rows
  int proj_dtype;
  long ld;
  int q_off, k_off, v_off;  // first column of the query, key (or forget gate) and value parts
  int mode;
  int H, dim, vdim;
  const float* decay;     // [H]                  FIXED_DECAY
  const float* inv_freq;  // [rot / 2]            FIXED_DECAY (may be null when rot == 0)
  int rot;
  float key_scale;
  int act;  // 1: silu on the raw query, key and value (FIXED_DECAY)
  const float* gate_bias;  // [H * dim]           FORGET_GATE, KEY_DECAY
  const float* lower;      // [H * dim]           FORGET_GATE
  const float* gate_map;   // [rank, H * dim]     KEY_DECAY
  int low_off, rank;       //                     KEY_DECAY
  float q_scale, power;    //                     KEY_DECAY
  const float* steps;      // [T, 2, H]           STEP_DECAY: factor on the value, decay
  const float* skip;       // [H]                 STEP_DECAY
  int heads_per_group;     //                     STEP_DECAY (1 otherwise)
  float* state;            // [slots, H, dim, vdim]
  const int* state_slot;   // [S]
  const int* q_start;      // [S + 1]
  const int* positions;    // [T]
  float* out;              // [T, ldo]: o_t at columns head * vdim + j
  long ldo;
  float* ready;          // [T, planes, H * dim] floats written by the first kernel (null: transform while staging)
  int slices;            // threads per column (a power of two, at most 32)
  int cols_per_block;    // threads / slices
  int tokens_per_round;
};

// sigmoid(z)^power by way of ln sigmoid(z) = -(ln(1 + e^-|z|) + max(-z, 0))
__device__ __forceinline__ float sigmoid_power(float z, float power) {
  return expf(-power * (log1pf(expf(-fabsf(z))) + fmaxf(-z, 0.f)));
}

// q_t, b_t and a_t of element (token, head, i) from the raw projection row, in 32-bit.
__device__ __forceinline__ void transform(const RecurrenceArgs& p, int token, int head, int i, float& qv,
                                          float& bv, float& av) {
  const size_t rowp = (size_t)token * p.ld;
  const size_t qo = rowp + p.q_off + (size_t)head * p.dim, ko = rowp + p.k_off + (size_t)head * p.dim;
  av = 0.f;
  if (p.mode == FIXED_DECAY) {
    qv = ld_any(p.proj, p.proj_dtype, qo + i);
    bv = ld_any(p.proj, p.proj_dtype, ko + i);
    if (p.act == 1) {
      qv = qv / (1.f + expf(-qv));
      bv = bv / (1.f + expf(-bv));
    }
    if (i < p.rot) {
      const int half = p.rot / 2;
      const int f = i < half ? i : i - half;
      const int other = i < half ? i + half : i - half;
      float sn, cs;
      sincosf((float)p.positions[token] * p.inv_freq[f], &sn, &cs);
      float q2 = ld_any(p.proj, p.proj_dtype, qo + other);
      float k2 = ld_any(p.proj, p.proj_dtype, ko + other);
      if (p.act == 1) {
        q2 = q2 / (1.f + expf(-q2));
        k2 = k2 / (1.f + expf(-k2));
      }
      // first of the pair: u cos - v sin; second: v cos + u sin
      qv = i < half ? qv * cs - q2 * sn : qv * cs + q2 * sn;
      bv = i < half ? bv * cs - k2 * sn : bv * cs + k2 * sn;
    }
    bv *= p.key_scale;
  } else if (p.mode == KEY_DECAY) {
    qv = ld_any(p.proj, p.proj_dtype, qo + i) * p.q_scale;
    bv = ld_any(p.proj, p.proj_dtype, ko + i) * p.key_scale;
    const int c = head * p.dim + i, hd = p.H * p.dim;
    float z = p.gate_bias[c];
    if (p.proj_dtype == DSP_F32) {
      const float* low = reinterpret_cast<const float*>(p.proj) + rowp + p.low_off;
#pragma unroll 8
      for (int r = 0; r < p.rank; ++r) z = fmaf(p.gate_map[(size_t)r * hd + c], low[r], z);
    } else {
      for (int r = 0; r < p.rank; ++r) z = fmaf(p.gate_map[(size_t)r * hd + c], ld_any(p.proj, p.proj_dtype, rowp + p.low_off + r), z);
    }
    av = sigmoid_power(z, p.power);
  } else {
    const float rq = ld_any(p.proj, p.proj_dtype, qo + i);
    qv = rq / (1.f + expf(-rq));
    const float rf = ld_any(p.proj, p.proj_dtype, ko + i) + p.gate_bias[head * p.dim + i];
    const float lo = p.lower[head * p.dim + i];
    av = lo + (1.f - lo) * (1.f / (1.f + expf(-rf)));
    bv = 1.f - av;
  }
}

// ready[t][0] = q, [1] = b, [2] = a (FORGET_GATE and KEY_DECAY), each [H * dim]
__global__ void __launch_bounds__(256) recurrence_prepare_kernel(const RecurrenceArgs p, int T) {
  const int hd = p.H * p.dim, planes = p.mode == FORGET_GATE ? 3 : 2;
  const long n = (long)T * hd;
  for (long idx = (long)blockIdx.x * blockDim.x + threadIdx.x; idx < n; idx += (long)gridDim.x * blockDim.x) {
    const int t = (int)(idx / hd), c = (int)(idx % hd);
    if (p.positions[t] < 0) continue;
    float qv, bv, av;
    transform(p, t, c / p.dim, c % p.dim, qv, bv, av);
    float* dst = p.ready + (size_t)t * planes * hd + c;
    dst[0] = qv;
    dst[hd] = bv;
    if (planes == 3) dst[2 * hd] = av;
  }
}

// The same for KEY_DECAY: a block takes LOW_TOKENS tokens and 256 channels, so that a row of the map
// is read once for all of its tokens (the same chain of sums as in `transform`).
constexpr int LOW_TOKENS = 8;
__global__ void __launch_bounds__(256) key_decay_prepare_kernel(const RecurrenceArgs p, int T) {
  extern __shared__ float low[];  // [LOW_TOKENS][rank]
  const int hd = p.H * p.dim, t0 = blockIdx.x * LOW_TOKENS, n = min(LOW_TOKENS, T - t0);
  for (int i = threadIdx.x; i < LOW_TOKENS * p.rank; i += blockDim.x) {
    const int k = i / p.rank;
    low[i] = k < n ? ld_any(p.proj, p.proj_dtype, (size_t)(t0 + k) * p.ld + p.low_off + i % p.rank) : 0.f;
  }
  __syncthreads();
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= hd) return;
  float z[LOW_TOKENS];
#pragma unroll
  for (int k = 0; k < LOW_TOKENS; ++k) z[k] = p.gate_bias[c];
  for (int r = 0; r < p.rank; ++r) {
    const float m = p.gate_map[(size_t)r * hd + c];
#pragma unroll
    for (int k = 0; k < LOW_TOKENS; ++k) z[k] = fmaf(m, low[k * p.rank + r], z[k]);
  }
#pragma unroll
  for (int k = 0; k < LOW_TOKENS; ++k) {
    if (k >= n || p.positions[t0 + k] < 0) continue;
    const size_t rowp = (size_t)(t0 + k) * p.ld;
    float* dst = p.ready + (size_t)(t0 + k) * 3 * hd + c;
    dst[0] = ld_any(p.proj, p.proj_dtype, rowp + p.q_off + c) * p.q_scale;
    dst[hd] = ld_any(p.proj, p.proj_dtype, rowp + p.k_off + c) * p.key_scale;
    dst[2 * hd] = sigmoid_power(z[k], p.power);
  }
}

__device__ __forceinline__ void cp_async4(float* smem, const float* gmem) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"((uint32_t)__cvta_generic_to_shared(smem)), "l"(gmem));
}

__device__ __forceinline__ void cp_async16(float* smem, const float* gmem) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((uint32_t)__cvta_generic_to_shared(smem)), "l"(gmem));
}

// The kernel for more than 256 state rows: a thread holds ROWS rows of one column.  ROWS: state rows a
// thread holds; TPR: tokens per staging round; KIND: what a_t is
template <int ROWS, int TPR, int KIND>
__global__ void __launch_bounds__(THREADS)
linear_recurrence_kernel(const RecurrenceArgs p) {
  extern __shared__ float smem[];
  const int seq = blockIdx.z, head = blockIdx.y;
  const int t0 = p.q_start[seq], t1 = p.q_start[seq + 1];
  if (t1 <= t0 || p.positions[t0] < 0) return;
  const int tid = threadIdx.x;
  const int slice = tid % p.slices, col_local = tid / p.slices;
  const int col = blockIdx.x * p.cols_per_block + col_local;
  const bool col_ok = col < p.vdim;
  const int dpad = p.slices * ROWS;  // state rows covered by the threads of a column (>= dim)
  constexpr int R = TPR;
  const int C = p.cols_per_block;
  constexpr bool gate = KIND == VECTOR_DECAY, per_token = KIND == TOKEN_DECAY;
  constexpr int planes = gate ? 3 : 2;
  // one staging buffer: [planes][R][dpad], v [R][C], per-token numbers [2][R]; two of them when rounds
  // arrive by cp.async
  const bool streamed = per_token || p.ready != nullptr;
  const int buf_floats = planes * R * dpad + R * C + (per_token ? 2 * R : 0);
  float* os = smem + (streamed ? 2 : 1) * buf_floats;  // [R][C]
  // row k of this thread's ROWS: four neighbours, then the next four behind all the slices' first fours
  auto row_of = [&](int k) { return (k >> 2) * (p.slices * 4) + slice * 4 + (k & 3); };

  float* sp = p.state + (((size_t)p.state_slot[seq] * p.H + head) * p.dim) * p.vdim;
  float S[ROWS];
#pragma unroll
  for (int k = 0; k < ROWS; ++k) {
    const int i = row_of(k);
    S[k] = (col_ok && i < p.dim) ? sp[(size_t)i * p.vdim + col] : 0.f;
  }
  const float decay = KIND == SCALAR_DECAY ? p.decay[head] : 0.f;
  const float skip = per_token ? p.skip[head] : 0.f;
  const int hd = p.H * p.dim;

  // rows beyond dim stay zero in every buffer: they are written here once and never again
  if (dpad > p.dim)
    for (int idx = tid; idx < (streamed ? 2 : 1) * buf_floats; idx += THREADS) smem[idx] = 0.f;
  __syncthreads();

  // rows of 16-byte pieces where every address allows it, single floats otherwise
  const float* rows = reinterpret_cast<const float*>(p.proj);
  const bool whole = p.ld % 4 == 0 && (((uintptr_t)rows) & 15) == 0;
  const bool wide = p.dim % 4 == 0 && (per_token ? whole && p.q_off % 4 == 0 && p.k_off % 4 == 0 : (((uintptr_t)p.ready) & 15) == 0);
  // values that need no arithmetic before the recurrence arrive by cp.async too
  const bool v_async = p.proj_dtype == DSP_F32 && p.act == 0;
  const bool v_wide = whole && p.v_off % 4 == 0 && p.vdim % 4 == 0 && C % 4 == 0;
  const int group0 = (head / p.heads_per_group) * p.dim;
  auto stage_async = [&](int base, float* buf) {
    const int n = min(R, t1 - base);
    for (int pl = 0; pl < planes; ++pl)
      for (int r = tid >> 5; r < n; r += THREADS / 32) {
        float* dst = buf + (pl * R + r) * dpad;
        const float* src = per_token ? rows + (size_t)(base + r) * p.ld + (pl == 0 ? p.q_off : p.k_off) + group0
                                     : p.ready + ((size_t)(base + r) * planes + pl) * hd + head * p.dim;
        if (wide)
          for (int i = (tid & 31) * 4; i < p.dim; i += 128) cp_async16(dst + i, src + i);
        else
          for (int i = tid & 31; i < p.dim; i += 32) cp_async4(dst + i, src + i);
      }
    if (v_async) {
      float* vs = buf + planes * R * dpad;
      const float* src = rows + p.v_off + (size_t)head * p.vdim;
      if (v_wide) {
        for (int idx = tid; idx < n * (C / 4); idx += THREADS) {
          const int r = idx / (C / 4), cl = (idx % (C / 4)) * 4, c = blockIdx.x * C + cl;
          if (c < p.vdim) cp_async16(vs + r * C + cl, src + (size_t)(base + r) * p.ld + c);
        }
      } else {
        for (int idx = tid; idx < n * C; idx += THREADS) {
          const int r = idx / C, c = blockIdx.x * C + idx % C;
          if (c < p.vdim) cp_async4(vs + idx, src + (size_t)(base + r) * p.ld + c);
        }
      }
    }
    if (per_token && tid < 2 * n)
      cp_async4(buf + planes * R * dpad + R * C + (tid & 1) * R + (tid >> 1), p.steps + ((size_t)(base + (tid >> 1)) * 2 + (tid & 1)) * p.H + head);
    asm volatile("cp.async.commit_group;\n");
  };
  auto stage_values = [&](int base, float* buf) {
    const int n = min(R, t1 - base);
    float* vs = buf + planes * R * dpad;
    for (int idx = tid; idx < n * C; idx += THREADS) {
      const int r = idx / C, c = blockIdx.x * C + idx % C;
      float v = c < p.vdim ? ld_any(p.proj, p.proj_dtype, (size_t)(base + r) * p.ld + p.v_off + (size_t)head * p.vdim + c) : 0.f;
      if (p.act == 1) v = v / (1.f + expf(-v));
      vs[idx] = v;
    }
  };

  if (streamed) stage_async(t0, smem);
  int turn = 0;
  for (int base = t0; base < t1; base += R, turn ^= 1) {
    const int n = min(R, t1 - base);
    float* buf = smem + (streamed ? turn : 0) * buf_floats;
    float* qs = buf;
    float* bs = buf + R * dpad;
    float* as = buf + 2 * R * dpad;
    float* vs = buf + planes * R * dpad;
    const float* steps = vs + R * C;
    if (streamed) {
      if (!v_async) stage_values(base, buf);
      if (base + R < t1) {
        stage_async(base + R, smem + (turn ^ 1) * buf_floats);
        asm volatile("cp.async.wait_group 1;\n");
      } else {
        asm volatile("cp.async.wait_group 0;\n");
      }
    } else {
      for (int idx = tid; idx < n * p.dim; idx += THREADS) {
        const int r = idx / p.dim, i = idx % p.dim;
        float qv, bv, av;
        transform(p, base + r, head, i, qv, bv, av);
        qs[r * dpad + i] = qv;
        bs[r * dpad + i] = bv;
        if (gate) as[r * dpad + i] = av;
      }
      stage_values(base, buf);
    }
    __syncthreads();
    auto one_token = [&](int r) {
      const float v = vs[r * C + col_local] * (per_token ? steps[r] : 1.f);
      const float a_all = per_token ? steps[R + r] : decay;
      const float* qr = qs + r * dpad + slice * 4;
      const float* br = bs + r * dpad + slice * 4;
      const float* ar = as + r * dpad + slice * 4;
      float acc0 = 0.f, acc1 = 0.f;
#pragma unroll
      for (int k = 0; k < ROWS; k += 4) {
        const int at = p.slices * k;
        const float4 q4 = *reinterpret_cast<const float4*>(qr + at), b4 = *reinterpret_cast<const float4*>(br + at);
        float4 a4 = make_float4(a_all, a_all, a_all, a_all);
        if (gate) a4 = *reinterpret_cast<const float4*>(ar + at);
        S[k] = fmaf(a4.x, S[k], b4.x * v);
        acc0 = fmaf(S[k], q4.x, acc0);
        S[k + 1] = fmaf(a4.y, S[k + 1], b4.y * v);
        acc1 = fmaf(S[k + 1], q4.y, acc1);
        S[k + 2] = fmaf(a4.z, S[k + 2], b4.z * v);
        acc0 = fmaf(S[k + 2], q4.z, acc0);
        S[k + 3] = fmaf(a4.w, S[k + 3], b4.w * v);
        acc1 = fmaf(S[k + 3], q4.w, acc1);
      }
      return acc0 + acc1;
    };
    // what goes out beside S^T q (read here, before the buffers turn)
    auto direct = [&](int r) { return per_token ? skip * vs[r * C + col_local] : 0.f; };
    if (n == R) {
      // a full round: the tokens' partial outputs first, then their reductions over the slices
      // side by side (the shuffles of one token do not wait for another's)
      float acc[R];
#pragma unroll
      for (int r = 0; r < R; ++r) acc[r] = one_token(r);
#pragma unroll
      for (int o = 1; o < 32; o <<= 1)
        if (o < p.slices) {
#pragma unroll
          for (int r = 0; r < R; ++r) acc[r] += __shfl_xor_sync(0xffffffffu, acc[r], o);
        }
      if (slice == 0) {
#pragma unroll
        for (int r = 0; r < R; ++r) os[r * C + col_local] = acc[r] + direct(r);
      }
    } else {
      for (int r = 0; r < n; ++r) {
        float acc = one_token(r);
        for (int o = 1; o < p.slices; o <<= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
        if (slice == 0) os[r * C + col_local] = acc + direct(r);
      }
    }
    __syncthreads();
    for (int idx = tid; idx < n * C; idx += THREADS) {
      const int r = idx / C, c = blockIdx.x * C + idx % C;
      if (c < p.vdim) p.out[(size_t)(base + r) * p.ldo + (size_t)head * p.vdim + c] = os[idx];
    }
  }
#pragma unroll
  for (int k = 0; k < ROWS; ++k) {
    const int i = row_of(k);
    if (col_ok && i < p.dim) sp[(size_t)i * p.vdim + col] = S[k];
  }
}

// Two 32-bit floats side by side: one instruction, each half rounded as its scalar form is.
typedef unsigned long long f32x2;
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

// The kernel for up to 256 state rows.  SLICES lanes, PAIRS pairs of rows a lane and PARTS groups of warps cover
// the state's rows (padded); every output is the sum of the groups' results, which meet in shared memory.
constexpr int TILE_STAGES = 3, BATCH = 8;

template <int SLICES, int PAIRS, int PARTS, int WARPS, bool STREAMED, int KIND>
struct Tile {
  static constexpr bool gate = KIND == VECTOR_DECAY, per_token = KIND == TOKEN_DECAY;
  static constexpr int planes = gate ? 3 : 2;
  static constexpr int part_rows = SLICES * 2 * PAIRS;                       // state rows of a group of warps
  static constexpr int rows = part_rows * PARTS;                             // state rows, padded
  static constexpr int cols = WARPS / PARTS * (32 / SLICES) * 4;             // value columns of a block
  static constexpr int round = rows <= 128 ? 16 : 8;                         // tokens staged together
  static constexpr int stage = planes * round * rows + round * cols + (per_token ? 2 * round : 0);
  static constexpr int meet = PARTS == 1 ? 0 : 2 * PARTS * round * cols;     // the groups' results of two rounds
  static constexpr int stages = STREAMED ? TILE_STAGES : 1;
  static constexpr size_t smem = sizeof(float) * (stages * stage + meet);
};

template <int SLICES, int PAIRS, int PARTS, int WARPS, bool STREAMED, int KIND>
__global__ void __launch_bounds__(32 * WARPS, 2)
recurrence_tile_kernel(const RecurrenceArgs p) {
  using L = Tile<SLICES, PAIRS, PARTS, WARPS, STREAMED, KIND>;
  constexpr bool gate = L::gate, per_token = L::per_token;
  constexpr int DP = L::rows, C = L::cols, R = L::round, planes = L::planes;
  extern __shared__ __align__(16) float tile_smem[];
  const int seq = blockIdx.z, head = blockIdx.y;
  const int t0 = p.q_start[seq], t1 = p.q_start[seq + 1];
  if (t1 <= t0 || p.positions[t0] < 0) return;
  const int tid = threadIdx.x, lane = tid & 31, slice = lane % SLICES;
  constexpr int TILE_THREADS = 32 * WARPS, PART_WARPS = WARPS / PARTS;
  const int part = (tid >> 5) / PART_WARPS;  // this warp's group of state rows
  const int cg = (tid >> 5) % PART_WARPS * (32 / SLICES) + lane / SLICES;  // this thread's group of four columns
  const int col0 = blockIdx.x * C + cg * 4;
  const float* rows = reinterpret_cast<const float*>(p.proj);
  const bool whole = p.ld % 4 == 0 && (((uintptr_t)rows) & 15) == 0;
  const bool wide = p.dim % 4 == 0 && (per_token ? whole && p.q_off % 4 == 0 && p.k_off % 4 == 0 : (((uintptr_t)p.ready) & 15) == 0);
  const bool v_async = p.proj_dtype == DSP_F32;
  const bool v_wide = whole && p.v_off % 4 == 0 && p.vdim % 4 == 0;
  const int hd = p.H * p.dim, group0 = (head / p.heads_per_group) * p.dim;

  // 2 PAIRS neighbouring state rows of columns col0 .. col0 + 3
  float* sp = p.state + (((size_t)p.state_slot[seq] * p.H + head) * p.dim) * p.vdim;
  const bool s_wide = p.vdim % 4 == 0;
  const int row0 = part * L::part_rows + slice * 2 * PAIRS;
  f32x2 S[PAIRS][4];  // [pair of rows 2k, 2k + 1][column]
#pragma unroll
  for (int k = 0; k < PAIRS; ++k) {
    float s[2][4] = {};
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int i = row0 + 2 * k + h;
      if (i >= p.dim || col0 >= p.vdim) continue;
      const float* src = sp + (size_t)i * p.vdim + col0;
      if (s_wide) {
        const float4 v = *reinterpret_cast<const float4*>(src);
        s[h][0] = v.x, s[h][1] = v.y, s[h][2] = v.z, s[h][3] = v.w;
      } else {
#pragma unroll
        for (int c = 0; c < 4; ++c)
          if (col0 + c < p.vdim) s[h][c] = src[c];
      }
    }
#pragma unroll
    for (int c = 0; c < 4; ++c) S[k][c] = pack2f(s[0][c], s[1][c]);
  }
  const float decay = KIND == SCALAR_DECAY ? p.decay[head] : 0.f;
  const float skip = per_token ? p.skip[head] : 0.f;

  // rows and columns beyond the head's own stay zero in every stage: written here and never again
  if (DP > p.dim || (int)(blockIdx.x + 1) * C > p.vdim) {
    for (int idx = tid; idx < L::stages * L::stage; idx += TILE_THREADS) tile_smem[idx] = 0.f;
    __syncthreads();
  }

  auto fill_values = [&](int base, float* buf) {  // values that need a conversion or an activation first
    const int n = min(R, t1 - base);
    float* vs = buf + planes * R * DP;
    for (int idx = tid; idx < n * C; idx += TILE_THREADS) {
      const int r = idx / C, c = blockIdx.x * C + idx % C;
      if (c >= p.vdim) continue;
      const float v = ld_any(p.proj, p.proj_dtype, (size_t)(base + r) * p.ld + p.v_off + (size_t)head * p.vdim + c);
      vs[idx] = p.act == 1 ? v / (1.f + expf(-v)) : v;
    }
  };
  auto stage_round = [&](int base, float* buf) {
    const int n = min(R, t1 - base);
    constexpr int ROW_THREADS = DP / 4 < 32 ? DP / 4 : 32;  // threads a row of one plane
#pragma unroll
    for (int pl = 0; pl < planes; ++pl)
      for (int r = tid / ROW_THREADS; r < n; r += TILE_THREADS / ROW_THREADS) {
        float* dst = buf + (pl * R + r) * DP;
        const float* src = per_token ? rows + (size_t)(base + r) * p.ld + (pl == 0 ? p.q_off : p.k_off) + group0
                                     : p.ready + ((size_t)(base + r) * planes + pl) * hd + head * p.dim;
#pragma unroll
        for (int i = (tid % ROW_THREADS) * 4; i < DP; i += ROW_THREADS * 4) {
          if (wide) {
            if (i < p.dim) cp_async16(dst + i, src + i);
          } else {
            for (int e = 0; e < 4; ++e)
              if (i + e < p.dim) cp_async4(dst + i + e, src + i + e);
          }
        }
      }
    float* vs = buf + planes * R * DP;
    if (v_async) {
      const float* src = rows + p.v_off + (size_t)head * p.vdim + blockIdx.x * C;
      for (int idx = tid; idx < n * (C / 4); idx += TILE_THREADS) {
        const int r = idx / (C / 4), c = (idx % (C / 4)) * 4, left = p.vdim - (int)blockIdx.x * C - c;
        if (v_wide) {
          if (left > 0) cp_async16(vs + r * C + c, src + (size_t)(base + r) * p.ld + c);
        } else {
          for (int e = 0; e < min(4, left); ++e) cp_async4(vs + r * C + c + e, src + (size_t)(base + r) * p.ld + c + e);
        }
      }
    } else {
      fill_values(base, buf);
    }
    if (per_token && tid < 2 * n)
      cp_async4(vs + R * C + (tid & 1) * R + (tid >> 1), p.steps + ((size_t)(base + (tid >> 1)) * 2 + (tid & 1)) * p.H + head);
  };

  float* meet = tile_smem + L::stages * L::stage;
  int turn2 = 0;  // which of the two meeting places the latest round used
  // one round; `full`: all of its tokens are there (no conditions between the tokens' loads)
  auto compute_round = [&](auto full, int base, const float* buf) {
    constexpr bool whole_round = decltype(full)::value;
    const int n = whole_round ? R : min(R, t1 - base);
    const float* vs = buf + planes * R * DP + cg * 4;
    const float* steps = buf + planes * R * DP + R * C;
    const float* qs = buf + row0;
    float* mine = meet + ((turn2 * PARTS + part) * R) * C + cg * 4;
#pragma unroll
    for (int r0 = 0; r0 < R; r0 += BATCH) {
      if (r0 >= n) break;
      float acc[BATCH * 4];
#pragma unroll
      for (int k = 0; k < BATCH; ++k) {
        const int r = r0 + k;
        float o[4] = {0.f, 0.f, 0.f, 0.f};
        if (whole_round || r < n) {
          const float4 v4 = *reinterpret_cast<const float4*>(vs + r * C);
          float v[4] = {v4.x, v4.y, v4.z, v4.w};
          float a_all = decay;
          if (per_token) {
            const float step = steps[r];
            a_all = steps[R + r];
#pragma unroll
            for (int c = 0; c < 4; ++c) v[c] *= step;
          }
          f32x2 v2[4], o2[4];
#pragma unroll
          for (int c = 0; c < 4; ++c) v2[c] = pack2f(v[c], v[c]);
          const f32x2 all2 = pack2f(a_all, a_all);
#pragma unroll
          for (int e = 0; e < PAIRS; ++e) {
            const f32x2* at = reinterpret_cast<const f32x2*>(qs + r * DP) + e;
            const f32x2 qe = at[0], be = at[R * DP / 2], ae = gate ? at[R * DP] : all2;
#pragma unroll
            for (int c = 0; c < 4; ++c) {
              f32x2& s = S[e][c];
              s = fma2(ae, s, mul2(be, v2[c]));
              o2[c] = e == 0 ? mul2(s, qe) : fma2(s, qe, o2[c]);
            }
          }
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            float even, odd;
            unpack2f(o2[c], even, odd);
            o[c] = even + odd;
          }
        }
#pragma unroll
        for (int c = 0; c < 4; ++c) acc[k * 4 + c] = o[c];
      }
      // sums over the slices: each exchange leaves a lane half of its values, and lane `slice` ends with values
      // slice * PER .. + PER - 1 of the BATCH * 4 (value k * 4 + c: token k, column c)
      constexpr int PER = BATCH * 4 / SLICES;
#pragma unroll
      for (int o = SLICES / 2, m = BATCH * 2; o > 0; o >>= 1, m >>= 1) {
        const bool upper = (lane & o) != 0;
#pragma unroll
        for (int i = 0; i < BATCH * 2; ++i)
          if (i < m) {
            const float keep = upper ? acc[i + m] : acc[i], give = upper ? acc[i] : acc[i + m];
            acc[i] = keep + __shfl_xor_sync(0xffffffffu, give, o);
          }
      }
#pragma unroll
      for (int i = 0; i < PER; ++i) {
        const int at = slice * PER + i, r = r0 + (at >> 2), c = at & 3;
        if (whole_round || r < n) {
          if (per_token && part == 0) acc[i] = fmaf(skip, vs[r * C + c], acc[i]);
          if (PARTS == 1 && col0 + c < p.vdim) p.out[(size_t)(base + r) * p.ldo + (size_t)head * p.vdim + col0 + c] = acc[i];
        }
      }
      if constexpr (PARTS > 1) {
        static_assert(PER == 4, "a lane ends with the four columns of one token");
        if (whole_round || r0 + slice < n)
          *reinterpret_cast<float4*>(mine + (r0 + slice) * C) = make_float4(acc[0], acc[1], acc[2], acc[3]);
      }
    }
  };

  auto compute = [&](int base, const float* buf) {
    turn2 ^= 1;
    if (base + R <= t1)
      compute_round(std::true_type{}, base, buf);
    else
      compute_round(std::false_type{}, base, buf);
  };

  // the outputs of the round at `base`, from what the groups of warps left (called behind a barrier)
  auto flush = [&](int base) {
    if constexpr (PARTS > 1) {
      const int n = min(R, t1 - base);
      const float* r0 = meet + turn2 * PARTS * R * C;
      for (int idx = tid; idx < n * C; idx += TILE_THREADS) {
        const int c = blockIdx.x * C + idx % C;
        float y = r0[idx];
#pragma unroll
        for (int k = 1; k < PARTS; ++k) y += r0[k * R * C + idx];
        if (c < p.vdim) p.out[(size_t)(base + idx / C) * p.ldo + (size_t)head * p.vdim + c] = y;
      }
    }
  };

  if constexpr (STREAMED) {
    for (int s = 0; s < TILE_STAGES - 1; ++s) {
      if (t0 + s * R < t1) stage_round(t0 + s * R, tile_smem + s * L::stage);
      asm volatile("cp.async.commit_group;\n");
    }
    int turn = 0;
    for (int base = t0; base < t1; base += R, turn = (turn + 1) % TILE_STAGES) {
      float* buf = tile_smem + turn * L::stage;
      asm volatile("cp.async.wait_group %0;\n" ::"n"(TILE_STAGES - 2));
      __syncthreads();  // this round has landed for everyone; the round before has been read by everyone
      if (base > t0) flush(base - R);
      const int ahead = base + (TILE_STAGES - 1) * R;
      if (ahead < t1) stage_round(ahead, tile_smem + ((turn + TILE_STAGES - 1) % TILE_STAGES) * L::stage);
      asm volatile("cp.async.commit_group;\n");
      if (v_async && p.act == 1) {  // the activation of the values, in place
        float* vs = buf + planes * R * DP;
        for (int idx = tid; idx < R * C; idx += TILE_THREADS) vs[idx] = vs[idx] / (1.f + expf(-vs[idx]));
        __syncthreads();
      }
      compute(base, buf);
    }
    asm volatile("cp.async.wait_group 0;\n");
  } else {
    for (int base = t0; base < t1; base += R) {
      const int n = min(R, t1 - base);
      __syncthreads();
      if (base > t0) flush(base - R);
      if (per_token) {
        stage_round(base, tile_smem);
        asm volatile("cp.async.commit_group;\n");
        asm volatile("cp.async.wait_group 0;\n");
        __syncthreads();
        compute(base, tile_smem);
        continue;
      }
      for (int idx = tid; idx < n * p.dim; idx += TILE_THREADS) {
        const int r = idx / p.dim, i = idx % p.dim;
        float qv, bv, av;
        transform(p, base + r, head, i, qv, bv, av);
        tile_smem[r * DP + i] = qv;
        tile_smem[(R + r) * DP + i] = bv;
        if (gate) tile_smem[(2 * R + r) * DP + i] = av;
      }
      fill_values(base, tile_smem);
      __syncthreads();
      compute(base, tile_smem);
    }
  }
  if constexpr (PARTS > 1) {
    __syncthreads();
    flush(t0 + (t1 - t0 - 1) / R * R);
  }
#pragma unroll
  for (int k = 0; k < PAIRS; ++k) {
    float s[2][4];
#pragma unroll
    for (int c = 0; c < 4; ++c) unpack2f(S[k][c], s[0][c], s[1][c]);
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int i = row0 + 2 * k + h;
      if (i >= p.dim || col0 >= p.vdim) continue;
      float* dst = sp + (size_t)i * p.vdim + col0;
      if (s_wide) {
        *reinterpret_cast<float4*>(dst) = make_float4(s[h][0], s[h][1], s[h][2], s[h][3]);
      } else {
#pragma unroll
        for (int c = 0; c < 4; ++c)
          if (col0 + c < p.vdim) dst[c] = s[h][c];
      }
    }
  }
}

template <int SLICES, int PAIRS, int PARTS, int WARPS, bool STREAMED, int KIND>
int launch_tile_kind(const RecurrenceArgs& a, int S, cudaStream_t stream) {
  using L = Tile<SLICES, PAIRS, PARTS, WARPS, STREAMED, KIND>;
  static bool configured = false;
  if (!configured) {
    DSP_CUDA(cudaFuncSetAttribute(recurrence_tile_kernel<SLICES, PAIRS, PARTS, WARPS, STREAMED, KIND>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                  (int)L::smem));
    configured = true;
  }
  const dim3 grid((a.vdim + L::cols - 1) / L::cols, a.H, S);
  recurrence_tile_kernel<SLICES, PAIRS, PARTS, WARPS, STREAMED, KIND><<<grid, 32 * WARPS, L::smem, stream>>>(a);
  DSP_CHECK_LAUNCH("dsp_linear_recurrence");
  return 0;
}

template <int SLICES, int PAIRS, int PARTS, int WARPS, bool STREAMED>
int launch_tile(const RecurrenceArgs& a, int S, cudaStream_t stream) {
  if (a.mode == STEP_DECAY) return launch_tile_kind<SLICES, PAIRS, PARTS, WARPS, STREAMED, TOKEN_DECAY>(a, S, stream);
  if (a.mode == FIXED_DECAY) return launch_tile_kind<SLICES, PAIRS, PARTS, WARPS, STREAMED, SCALAR_DECAY>(a, S, stream);
  return launch_tile_kind<SLICES, PAIRS, PARTS, WARPS, STREAMED, VECTOR_DECAY>(a, S, stream);
}

template <int ROWS, int TPR, int KIND>
int launch_kind(const RecurrenceArgs& a, int S, size_t smem, cudaStream_t stream) {
  static size_t configured = 48 * 1024;
  if (smem > configured) {
    DSP_CUDA(cudaFuncSetAttribute(linear_recurrence_kernel<ROWS, TPR, KIND>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    configured = smem;
  }
  dim3 grid((a.vdim + a.cols_per_block - 1) / a.cols_per_block, a.H, S);
  linear_recurrence_kernel<ROWS, TPR, KIND><<<grid, THREADS, smem, stream>>>(a);
  DSP_CHECK_LAUNCH("dsp_linear_recurrence");
  return 0;
}

template <int ROWS, int TPR>
int launch(const RecurrenceArgs& a, int S, size_t smem, cudaStream_t stream) {
  if (a.mode == STEP_DECAY) return launch_kind<ROWS, TPR, TOKEN_DECAY>(a, S, smem, stream);
  if (a.mode == FIXED_DECAY) return launch_kind<ROWS, TPR, SCALAR_DECAY>(a, S, smem, stream);
  return launch_kind<ROWS, TPR, VECTOR_DECAY>(a, S, smem, stream);
}
}  // namespace

// scratch: null (one kernel, tokens transformed as they are staged) or room for [T, planes, H * dim]
// floats, planes = 2 with one decay for all rows, else 3 (a first kernel transforms every token, the
// recurrence streams); STEP_DECAY takes none.
extern "C" int dsp_linear_recurrence(const void* proj, int proj_dtype, long ld, int q_off, int k_off,
                                     int v_off, int mode, int H, int dim, int vdim, const float* decay,
                                     const float* inv_freq, int rot, float key_scale, int act,
                                     const float* gate_bias, const float* lower,
                                     const float* gate_map, int low_off, int rank, float q_scale, float power,
                                     const float* steps, const float* skip, int heads_per_group, float* state,
                                     const int* state_slot, const int* q_start, const int* positions,
                                     float* out, long ldo, int S, int T, float* scratch, cudaStream_t stream) {
  if (S == 0 || T == 0) return 0;
  DSP_REQUIRE(proj && state && state_slot && q_start && positions && out, "dsp_linear_recurrence: missing operand");
  DSP_REQUIRE(H > 0 && H <= 65535 && S <= 65535, "dsp_linear_recurrence: H=%d, S=%d outside the grid", H, S);
  DSP_REQUIRE(dim > 0 && dim <= 1024 && vdim > 0, "dsp_linear_recurrence: dim=%d (at most 1024), vdim=%d", dim, vdim);
  if (mode == FIXED_DECAY) {
    DSP_REQUIRE(decay != nullptr, "dsp_linear_recurrence: no decay");
    DSP_REQUIRE(rot >= 0 && rot <= dim && rot % 2 == 0 && (rot == 0 || inv_freq), "dsp_linear_recurrence: rot=%d", rot);
    DSP_REQUIRE(act == 0 || act == 1, "dsp_linear_recurrence: unknown activation %d", act);
  } else if (mode == FORGET_GATE) {
    DSP_REQUIRE(gate_bias && lower, "dsp_linear_recurrence: no gate bias or lower bound");
  } else if (mode == KEY_DECAY) {
    DSP_REQUIRE(gate_bias && gate_map && rank > 0 && rank <= 1024, "dsp_linear_recurrence: no decay map or bias, or rank %d outside 1..1024", rank);
  } else if (mode == STEP_DECAY) {
    DSP_REQUIRE(steps && skip && proj_dtype == DSP_F32 && !scratch, "dsp_linear_recurrence: no step sizes, or rows that are not floats");
    DSP_REQUIRE(heads_per_group > 0 && H % heads_per_group == 0, "dsp_linear_recurrence: %d heads in groups of %d", H, heads_per_group);
  } else {
    DSP_REQUIRE(false, "dsp_linear_recurrence: unknown mode %d", mode);
  }
  RecurrenceArgs a;
  a.proj = proj; a.proj_dtype = proj_dtype; a.ld = ld;
  a.q_off = q_off; a.k_off = k_off; a.v_off = v_off; a.mode = mode;
  a.H = H; a.dim = dim; a.vdim = vdim;
  a.decay = decay; a.inv_freq = inv_freq; a.rot = rot; a.key_scale = key_scale; a.act = mode == FIXED_DECAY ? act : 0;
  a.gate_bias = gate_bias; a.lower = lower;
  a.gate_map = gate_map; a.low_off = low_off; a.rank = rank; a.q_scale = q_scale; a.power = power;
  a.steps = steps; a.skip = skip; a.heads_per_group = mode == STEP_DECAY ? heads_per_group : 1;
  a.state = state; a.state_slot = state_slot; a.q_start = q_start; a.positions = positions;
  a.out = out; a.ldo = ldo; a.ready = scratch;
  // one column a thread, 32 threads a column, 16 or 32 state rows a thread (beyond 256 state rows)
  const bool tiled = dim <= 256;
  const int slices = 32, rows = (dim + slices - 1) / slices;
  a.slices = slices;
  a.cols_per_block = THREADS / slices;
  const int R = rows <= 16 ? 16 : 32;
  const int dpad = slices * R;
  a.tokens_per_round = 8;
  const int planes = mode == FORGET_GATE || mode == KEY_DECAY ? 3 : 2;
  const size_t buf = (size_t)planes * a.tokens_per_round * dpad + (size_t)a.tokens_per_round * a.cols_per_block +
                     (mode == STEP_DECAY ? 2 * a.tokens_per_round : 0);
  const size_t smem = sizeof(float) * ((scratch || mode == STEP_DECAY ? 2 : 1) * buf + (size_t)a.tokens_per_round * a.cols_per_block);
  DSP_REQUIRE(tiled || smem <= 227 * 1024, "dsp_linear_recurrence: state rows of %d do not fit shared memory", dim);
  if (scratch && mode == KEY_DECAY) {
    const unsigned tiles = (unsigned)((H * dim + 255) / 256);
    DSP_REQUIRE(tiles <= 65535, "dsp_linear_recurrence: %d heads of %d are too many", H, dim);
    key_decay_prepare_kernel<<<dim3((T + LOW_TOKENS - 1) / LOW_TOKENS, tiles), 256, sizeof(float) * LOW_TOKENS * rank, stream>>>(a, T);
    DSP_CHECK_LAUNCH("dsp_linear_recurrence (first kernel)");
  } else if (scratch) {
    const long n = (long)T * H * dim;
    const int sms = dsp_num_sms();
    const long want = (n + 255) / 256, cap = (long)(sms > 0 ? sms : 148) * 8;
    recurrence_prepare_kernel<<<(unsigned)(want < cap ? want : cap), 256, 0, stream>>>(a, T);
    DSP_CHECK_LAUNCH("dsp_linear_recurrence (first kernel)");
  }
  if (scratch || (mode == STEP_DECAY && T > 2 * S)) {  // portions of prompts
    if (dim <= 32) return launch_tile<8, 1, 2, 8, true>(a, S, stream);
    if (dim <= 64) return launch_tile<8, 1, 4, 8, true>(a, S, stream);
    if (dim <= 128) return launch_tile<8, 1, 8, 8, true>(a, S, stream);
    if (tiled) return launch_tile<8, 2, 8, 8, true>(a, S, stream);
  } else {  // single tokens
    if (dim <= 32) return launch_tile<8, 2, 1, 4, false>(a, S, stream);
    if (dim <= 64) return launch_tile<16, 2, 1, 4, false>(a, S, stream);
    if (dim <= 128) return launch_tile<32, 2, 1, 4, false>(a, S, stream);
    if (tiled) return launch_tile<32, 4, 1, 4, false>(a, S, stream);
  }
  if (R == 16) return launch<16, 8>(a, S, smem, stream);
  return launch<32, 8>(a, S, smem, stream);
}
