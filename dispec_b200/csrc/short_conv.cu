// Short causal convolutions over time, channel by channel, with the last taps - 1 inputs of every
// request kept in its state slot (32-bit floats, zeros at admission):
//
//     y_t[c] = sum_j w[j][c] * u_(t - taps + 1 + j)[c]          (w float [taps, channels])
//
// where u are columns of the rows of a mixer's fused projection (float or bfloat16).  Three users:
//
//   dsp_conv_steps             y, plus a bias, through silu, as float rows [T, channels]; and, for a state-space
//                              recurrence, per token and head step = softplus(raw + bias) and decay =
//                              exp(-exp(A_log) * step) as `steps` [T, 2, heads].
//   dsp_qkv_conv_rotate_store  y over the columns [q (H x Dk) | k (G x Dk) | v (G x Dv)], then queries and keys
//                              turned by position * inv_freq[i], pairs (2i, 2i + 1) or (i, i + rot/2), then
//                              divided by their root mean square per head (eps inside the root, no
//                              weight) if asked for; queries go to q_out, keys and values (times
//                              v_scale) to the pages.
//   dsp_conv_heads             silu(y) over the columns [A heads of dim | B heads of dim | H heads of vdim] as float rows,
//                              the first two kinds of heads divided by their length, x / sqrt(sum(x^2) + eps), the
//                              first one then times a factor; and, for a delta rule, per token and head
//                              sigmoid(raw b) and -exp(A_log) * softplus(raw a + bias) as `steps` [T, 2, H].  A warp takes
//                              one head of one token, or of four neighbouring ones in steps with portions of prompts.
//
// Every token has a block (or a row of blocks) of its own: its taps come from the rows of the step, and,
// before the first token the step brings for the request, from the state slot.  The block of that
// first token is the only one that touches the slot: it also computes the tokens 1 .. taps - 2, which would
// have to read it too, and then leaves the step's last taps - 1 inputs there, which it takes from
// the projection's rows, not from other blocks.  A thread keeps to its own channels throughout, so
// within the block nothing is ordered by barriers.  Rows with a negative position (padding of a captured
// step) are skipped: their state slot belongs to someone else.
#include "common.cuh"

namespace {

struct ConvIn {
  const void* u;  // [T, ld], first convolved column at `off`
  int dtype;
  long ld;
  int off, channels, taps;
  const float* w;  // [taps, channels] (null: taps == 1 and y = u)
  float* hist;     // [slots, taps - 1, channels]
  const int* state_slot;
  const int* q_start;
  const int* seq_of_token;
  const int* positions;
};

// What a block of token t does: its first local token, how many, and whether it owns the state slot.
struct Turn {
  int seq, first, count, n, row0;
  bool owner;
};
__device__ __forceinline__ Turn turn_of(const ConvIn& c, int t) {
  Turn r;
  r.seq = c.seq_of_token[t];
  r.row0 = c.q_start[r.seq];
  r.n = c.q_start[r.seq + 1] - r.row0;
  const int i = t - r.row0;
  r.first = i;
  r.owner = i == 0;
  r.count = i == 0 ? min(r.n, max(1, c.taps - 1)) : (i < c.taps - 1 ? 0 : 1);
  return r;
}

// input of channel c at local token j of the request's portion (negative: from the state slot)
__device__ __forceinline__ float input_at(const ConvIn& p, const Turn& r, const float* hist, int c, int j) {
  if (j >= 0) return ld_any(p.u, p.dtype, (size_t)(r.row0 + j) * p.ld + p.off + c);
  return hist[(size_t)(p.taps - 1 + j) * p.channels + c];
}

__device__ __forceinline__ float conv_at(const ConvIn& p, const Turn& r, const float* hist, int c, int i) {
  if (!p.w) return input_at(p, r, hist, c, i);
  float acc = 0.f;
  for (int j = 0; j < p.taps; ++j) acc = fmaf(p.w[(size_t)j * p.channels + c], input_at(p, r, hist, c, i - p.taps + 1 + j), acc);
  return acc;
}

// four neighbouring channels of a token whose taps all lie in the step's rows (floats, 16-byte aligned): the
// same sums in the same order
__device__ __forceinline__ float4 conv_at4(const ConvIn& p, const float* row, int c) {
  const float* u = row + p.off + c - (size_t)(p.taps - 1) * p.ld;
  float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
  for (int j = 0; j < p.taps; ++j) {
    const float4 w = *reinterpret_cast<const float4*>(p.w + (size_t)j * p.channels + c);
    const float4 x = *reinterpret_cast<const float4*>(u + (size_t)j * p.ld);
    acc.x = fmaf(w.x, x.x, acc.x);
    acc.y = fmaf(w.y, x.y, acc.y);
    acc.z = fmaf(w.z, x.z, acc.z);
    acc.w = fmaf(w.w, x.w, acc.w);
  }
  return acc;
}
// whether rows, weights and slots can be taken four channels at a time
__device__ __forceinline__ bool in_fours(const ConvIn& p) {
  return p.w && p.dtype == DSP_F32 && p.channels % 4 == 0 && p.off % 4 == 0 && p.ld % 4 == 0 &&
         (((uintptr_t)p.u | (uintptr_t)p.w | (uintptr_t)p.hist) & 15) == 0;
}

// A portion of one token (decoding): four neighbouring channels' convolution and the new state in one
// pass, every load issued before the first value is used.  The same sums in the same order.
constexpr int SINGLE_TAPS = 8;
__device__ __forceinline__ bool is_single(const ConvIn& p, const Turn& r) {
  return r.n == 1 && p.taps > 1 && p.taps <= SINGLE_TAPS && in_fours(p);
}
__device__ __forceinline__ float4 conv_single4(const ConvIn& p, const float* row, float* hist, int c) {
  float4 x[SINGLE_TAPS], acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int j = 0; j < SINGLE_TAPS; ++j)
    if (j < p.taps)
      x[j] = *reinterpret_cast<const float4*>(j < p.taps - 1 ? hist + (size_t)j * p.channels + c : row + p.off + c);
#pragma unroll
  for (int j = 0; j < SINGLE_TAPS; ++j)
    if (j < p.taps) {
      const float4 w = *reinterpret_cast<const float4*>(p.w + (size_t)j * p.channels + c);
      acc.x = fmaf(w.x, x[j].x, acc.x);
      acc.y = fmaf(w.y, x[j].y, acc.y);
      acc.z = fmaf(w.z, x[j].z, acc.z);
      acc.w = fmaf(w.w, x[j].w, acc.w);
    }
#pragma unroll
  for (int j = 1; j < SINGLE_TAPS; ++j)
    if (j < p.taps) *reinterpret_cast<float4*>(hist + (size_t)(j - 1) * p.channels + c) = x[j];
  return acc;
}

// leaves the portion's last taps - 1 inputs of channel c in the slot (in place: row m is written before
// the rows behind it are, and reads rows at or behind m + n)
__device__ __forceinline__ void keep_inputs(const ConvIn& p, const Turn& r, float* hist, int c) {
  for (int m = 0; m < p.taps - 1; ++m)
    hist[(size_t)m * p.channels + c] = input_at(p, r, hist, c, r.n - (p.taps - 1) + m);
}

__device__ __forceinline__ float softplus_f(float v) { return v > 20.f ? v + log1pf(expf(-v)) : log1pf(expf(v)); }

constexpr int PER_THREAD = 4;

__global__ void __launch_bounds__(256)
conv_steps_kernel(const ConvIn p, const float* __restrict__ bias, float* __restrict__ out, long ldo, int step_off,
                  int heads, const float* __restrict__ step_bias, const float* __restrict__ a_log,
                  float* __restrict__ steps) {
  const int t = blockIdx.x;
  if (p.positions[t] < 0) return;
  const Turn r = turn_of(p, t);
  float* hist = p.hist + (size_t)p.state_slot[r.seq] * (p.taps - 1) * p.channels;
  auto silu = [](float v) { return v / (1.f + expf(-v)); };
  const bool single = is_single(p, r);
  if ((single || (!r.owner && r.count == 1 && in_fours(p))) && ldo % 4 == 0 && ((uintptr_t)out & 15) == 0 && ((uintptr_t)bias & 15) == 0) {
    const int c = (blockIdx.y * 256 + threadIdx.x) * 4;
    if (c < p.channels) {
      const float* row = reinterpret_cast<const float*>(p.u) + (size_t)t * p.ld;
      float4 v = single ? conv_single4(p, row, hist, c) : conv_at4(p, row, c);
      if (bias) {
        const float4 b = *reinterpret_cast<const float4*>(bias + c);
        v.x += b.x, v.y += b.y, v.z += b.z, v.w += b.w;
      }
      *reinterpret_cast<float4*>(out + (size_t)t * ldo + c) = make_float4(silu(v.x), silu(v.y), silu(v.z), silu(v.w));
    }
  } else {
    for (int i = r.first; i < r.first + r.count; ++i)
#pragma unroll
      for (int k = 0; k < PER_THREAD; ++k) {
        const int c = (blockIdx.y * PER_THREAD + k) * 256 + threadIdx.x;
        if (c >= p.channels) break;
        out[(size_t)(r.row0 + i) * ldo + c] = silu(conv_at(p, r, hist, c, i) + (bias ? bias[c] : 0.f));
      }
    if (r.owner)
      for (int k = 0; k < PER_THREAD; ++k) {
        const int c = (blockIdx.y * PER_THREAD + k) * 256 + threadIdx.x;
        if (c < p.channels) keep_inputs(p, r, hist, c);
      }
  }
  if (blockIdx.y == 0)
    for (int h = threadIdx.x; h < heads; h += blockDim.x) {
      const float step = softplus_f(ld_any(p.u, p.dtype, (size_t)t * p.ld + step_off + h) + step_bias[h]);
      steps[((size_t)t * 2) * heads + h] = step;
      steps[((size_t)t * 2 + 1) * heads + h] = expf(-expf(a_log[h]) * step);
    }
}

__global__ void __launch_bounds__(256)
qkv_conv_rotate_store_kernel(const ConvIn p, const int* __restrict__ page_table, int pt_stride, void* __restrict__ k_pool,
                             void* __restrict__ v_pool, int pool_dtype, const float* __restrict__ inv_freq, int rot,
                             int interleaved, int head_norm, float norm_eps, float v_scale, void* __restrict__ q_out,
                             long ld_q, int H, int G, int Dk, int Dv, int page_size, int num_pages, int write_kv, int* err) {
  extern __shared__ __align__(16) float row[];  // [channels] then [rot/2] cosines, [rot/2] sines
  const int t = blockIdx.x;
  if (p.positions[t] < 0) return;
  const Turn r = turn_of(p, t);
  if (r.count == 0) return;
  float* hist = p.taps > 1 ? p.hist + (size_t)p.state_slot[r.seq] * (p.taps - 1) * p.channels : nullptr;
  float* cs = row + p.channels;
  const bool single = is_single(p, r);
  const int half = rot / 2, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, warps = blockDim.x >> 5;
  for (int i = r.first; i < r.first + r.count; ++i) {
    const int tok = r.row0 + i, pos = p.positions[tok];
    if (single || (in_fours(p) && i >= p.taps - 1)) {
      const float* u = reinterpret_cast<const float*>(p.u) + (size_t)tok * p.ld;
      for (int c = tid * 4; c < p.channels; c += blockDim.x * 4)
        *reinterpret_cast<float4*>(row + c) = single ? conv_single4(p, u, hist, c) : conv_at4(p, u, c);
    } else
      for (int c = tid; c < p.channels; c += blockDim.x) row[c] = conv_at(p, r, hist, c, i);
    for (int m = tid; m < half; m += blockDim.x) sincosf((float)pos * inv_freq[m], &cs[half + m], &cs[m]);
    __syncthreads();
    const int page = write_kv ? page_table[(size_t)r.seq * pt_stride + pos / page_size] : -1;
    const bool store = write_kv && page >= 0 && page < num_pages;
    if (write_kv && !store && tid == 0) atomicOr(err, DSP_ERR_BAD_PAGE);
    const size_t at = (size_t)page * G * page_size + pos % page_size;  // (used only when `store`)
    for (int h = warp; h < H + G; h += warps) {
      float* x = row + h * Dk;
      for (int m = lane; m < half; m += 32) {
        const int a = interleaved ? 2 * m : m, b = interleaved ? 2 * m + 1 : m + half;
        const float u = x[a], v = x[b], c = cs[m], s = cs[half + m];
        x[a] = u * c - v * s;
        x[b] = v * c + u * s;
      }
      __syncwarp();
      float f = 1.f;
      if (head_norm) {
        float ss = 0.f;
        for (int d = lane; d < Dk; d += 32) ss = fmaf(x[d], x[d], ss);
        f = 1.f / sqrtf(warp_sum(ss) / (float)Dk + norm_eps);
      }
      if (h < H) {
        for (int d = lane; d < Dk; d += 32) st_any(q_out, pool_dtype, (size_t)tok * ld_q + (size_t)h * Dk + d, x[d] * f);
      } else if (store) {
        for (int d = lane; d < Dk; d += 32) st_any(k_pool, pool_dtype, (at + (size_t)(h - H) * page_size) * Dk + d, x[d] * f);
      }
    }
    if (store) {
      const float* v = row + (H + G) * Dk;
      for (int idx = tid; idx < G * Dv; idx += blockDim.x)
        st_any(v_pool, pool_dtype, (at + (size_t)(idx / Dv) * page_size) * Dv + idx % Dv, v[idx] * v_scale);
    }
    __syncthreads();  // the row is taken again
  }
  if (r.owner && p.taps > 1 && !single)
    for (int c = tid; c < p.channels; c += blockDim.x) keep_inputs(p, r, hist, c);
}

// One warp a (token or TOK tokens, head); blockIdx.y counts the heads, the last one stands for the steps.
constexpr int HEAD_WARPS = 8, HEAD_QUADS = 2;  // HEAD_QUADS: groups of four channels a lane keeps in registers

// one token: c0, n: the head's columns
__device__ __forceinline__ void conv_head_token(const ConvIn& p, int t, int lane, int c0, int n, bool unit, float factor, float eps,
                                                float* __restrict__ out, long ldo) {
  if (p.positions[t] < 0) return;
  const Turn r = turn_of(p, t);
  if (r.count == 0) return;
  float* hist = p.taps > 1 ? p.hist + (size_t)p.state_slot[r.seq] * (p.taps - 1) * p.channels : nullptr;
  auto silu = [](float v) { return v / (1.f + expf(-v)); };
  const bool single = is_single(p, r);
  if ((single || (!r.owner && r.count == 1 && in_fours(p))) && n % 4 == 0 && c0 % 4 == 0 && n <= 128 * HEAD_QUADS && ldo % 4 == 0 &&
      ((uintptr_t)out & 15) == 0) {
    const float* row = reinterpret_cast<const float*>(p.u) + (size_t)t * p.ld;
    float4 y[HEAD_QUADS];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < HEAD_QUADS; ++k) {
      const int i = (lane + 32 * k) * 4;
      if (i >= n) break;
      const float4 v = single ? conv_single4(p, row, hist, c0 + i) : conv_at4(p, row, c0 + i);
      y[k] = make_float4(silu(v.x), silu(v.y), silu(v.z), silu(v.w));
      ss += (y[k].x * y[k].x + y[k].y * y[k].y) + (y[k].z * y[k].z + y[k].w * y[k].w);
    }
    const float f = unit ? factor / sqrtf(warp_sum(ss) + eps) : 1.f;
#pragma unroll
    for (int k = 0; k < HEAD_QUADS; ++k) {
      const int i = (lane + 32 * k) * 4;
      if (i < n) *reinterpret_cast<float4*>(out + (size_t)t * ldo + c0 + i) = make_float4(y[k].x * f, y[k].y * f, y[k].z * f, y[k].w * f);
    }
    return;
  }
  for (int i = r.first; i < r.first + r.count; ++i) {
    float* dst = out + (size_t)(r.row0 + i) * ldo + c0;
    float ss = 0.f;
    for (int c = lane; c < n; c += 32) {
      const float y = silu(conv_at(p, r, hist, c0 + c, i));
      dst[c] = y;
      ss = fmaf(y, y, ss);
    }
    if (!unit) continue;
    const float f = factor / sqrtf(warp_sum(ss) + eps);
    for (int c = lane; c < n; c += 32) dst[c] *= f;
  }
  if (r.owner && p.taps > 1)
    for (int c = lane; c < n; c += 32) keep_inputs(p, r, hist, c0 + c);
}

// TOK neighbouring tokens of one request whose taps all lie in the step's rows: a row is loaded once for all of them,
// the weights once (the same sums in the same order)
template <int TAPS, int TOK>
__device__ __forceinline__ void conv_head_run(const ConvIn& p, int t, int lane, int c0, int n, bool unit, float factor, float eps,
                                              float* __restrict__ out, long ldo) {
  float4 y[TOK][HEAD_QUADS];
  float ss[TOK] = {};
  auto silu = [](float v) { return v / (1.f + expf(-v)); };
#pragma unroll
  for (int k = 0; k < HEAD_QUADS; ++k) {
    const int i = (lane + 32 * k) * 4;
    if (i >= n) break;
    const float* u = reinterpret_cast<const float*>(p.u) + (size_t)(t - (TAPS - 1)) * p.ld + c0 + i;
    float4 x[TOK + TAPS - 1], w[TAPS];
#pragma unroll
    for (int j = 0; j < TOK + TAPS - 1; ++j) x[j] = *reinterpret_cast<const float4*>(u + (size_t)j * p.ld);
#pragma unroll
    for (int j = 0; j < TAPS; ++j) w[j] = *reinterpret_cast<const float4*>(p.w + (size_t)j * p.channels + c0 + i);
#pragma unroll
    for (int m = 0; m < TOK; ++m) {
      float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int j = 0; j < TAPS; ++j) {
        a.x = fmaf(w[j].x, x[m + j].x, a.x);
        a.y = fmaf(w[j].y, x[m + j].y, a.y);
        a.z = fmaf(w[j].z, x[m + j].z, a.z);
        a.w = fmaf(w[j].w, x[m + j].w, a.w);
      }
      y[m][k] = make_float4(silu(a.x), silu(a.y), silu(a.z), silu(a.w));
      ss[m] += (y[m][k].x * y[m][k].x + y[m][k].y * y[m][k].y) + (y[m][k].z * y[m][k].z + y[m][k].w * y[m][k].w);
    }
  }
#pragma unroll
  for (int m = 0; m < TOK; ++m) {
    const float f = unit ? factor / sqrtf(warp_sum(ss[m]) + eps) : 1.f;
#pragma unroll
    for (int k = 0; k < HEAD_QUADS; ++k) {
      const int i = (lane + 32 * k) * 4;
      if (i < n) *reinterpret_cast<float4*>(out + (size_t)(t + m) * ldo + c0 + i) = make_float4(y[m][k].x * f, y[m][k].y * f, y[m][k].z * f, y[m][k].w * f);
    }
  }
}

template <int TOK>
__global__ void __launch_bounds__(32 * HEAD_WARPS)
conv_heads_kernel(const ConvIn p, int T, int A, int B, int dim, int vdim, float eps, float a_scale, float* __restrict__ out,
                  long ldo, int b_off, int a_off, int H, const float* __restrict__ step_bias,
                  const float* __restrict__ a_log, float* __restrict__ steps) {
  const int t = (blockIdx.x * HEAD_WARPS + (threadIdx.x >> 5)) * TOK, lane = threadIdx.x & 31, head = blockIdx.y;
  if (t >= T) return;
  const int end = min(T, t + TOK);
  if (head == A + B + H) {
    for (int idx = lane; idx < (end - t) * H; idx += 32) {
      const int tok = t + idx / H, h = idx % H;
      if (p.positions[tok] < 0) continue;
      steps[(size_t)tok * 2 * H + h] = 1.f / (1.f + expf(-ld_any(p.u, p.dtype, (size_t)tok * p.ld + b_off + h)));
      steps[((size_t)tok * 2 + 1) * H + h] = -expf(a_log[h]) * softplus_f(ld_any(p.u, p.dtype, (size_t)tok * p.ld + a_off + h) + step_bias[h]);
    }
    return;
  }
  const bool unit = head < A + B;
  const int c0 = unit ? head * dim : (A + B) * dim + (head - A - B) * vdim, n = unit ? dim : vdim;
  const float factor = head < A ? a_scale : 1.f;
  if (TOK > 1 && end == t + TOK && p.taps >= 2 && p.taps <= 4 && n % 4 == 0 && c0 % 4 == 0 && n <= 128 * HEAD_QUADS && in_fours(p) &&
      ldo % 4 == 0 && ((uintptr_t)out & 15) == 0) {
    const int seq = p.seq_of_token[t];
    if (p.positions[t] >= 0 && p.seq_of_token[end - 1] == seq && t - p.q_start[seq] >= p.taps - 1) {
      if (p.taps == 4) conv_head_run<4, TOK>(p, t, lane, c0, n, unit, factor, eps, out, ldo);
      else if (p.taps == 3) conv_head_run<3, TOK>(p, t, lane, c0, n, unit, factor, eps, out, ldo);
      else conv_head_run<2, TOK>(p, t, lane, c0, n, unit, factor, eps, out, ldo);
      return;
    }
  }
  for (int tok = t; tok < end; ++tok) conv_head_token(p, tok, lane, c0, n, unit, factor, eps, out, ldo);
}

int check(const ConvIn& p, const char* name) {
  DSP_REQUIRE(p.u && p.q_start && p.seq_of_token && p.positions && p.channels > 0, "%s: missing operand", name);
  DSP_REQUIRE(p.taps >= 1 && (p.taps == 1 || (p.w && p.hist && p.state_slot)), "%s: %d taps without weights or state", name, p.taps);
  return 0;
}
}  // namespace

extern "C" int dsp_conv_steps(const void* u, int dtype, long ld, int off, int channels, int taps, const float* w,
                              const float* bias, float* hist, const int* state_slot, const int* q_start,
                              const int* seq_of_token, const int* positions, float* out, long ldo, int step_off, int heads,
                              const float* step_bias, const float* a_log, float* steps, int T, cudaStream_t stream) {
  if (T == 0) return 0;
  const ConvIn p = {u, dtype, ld, off, channels, taps, w, hist, state_slot, q_start, seq_of_token, positions};
  if (const int rc = check(p, "dsp_conv_steps")) return rc;
  DSP_REQUIRE(out && w && state_slot && (heads == 0 || (step_bias && a_log && steps)), "dsp_conv_steps: missing operand");
  const int tiles = (channels + 256 * PER_THREAD - 1) / (256 * PER_THREAD);
  DSP_REQUIRE(tiles <= 65535, "dsp_conv_steps: %d channels are too many", channels);
  DSP_CUDA(launch_plain(conv_steps_kernel, dim3(T, tiles), dim3(256), 0, stream, p, bias, out, ldo, step_off, heads,
                        step_bias, a_log, steps));
  DSP_CHECK_LAUNCH("dsp_conv_steps");
  return 0;
}

extern "C" int dsp_qkv_conv_rotate_store(const void* u, int dtype, long ld, int taps, const float* w, float* hist,
                                         const int* state_slot, const int* q_start, const int* seq_of_token,
                                         const int* positions, const int* page_table, int pt_stride, void* k_pool,
                                         void* v_pool, int pool_dtype, const float* inv_freq, int rot, int interleaved,
                                         int head_norm, float norm_eps, float v_scale, void* q_out, long ld_q, int T, int H,
                                         int G, int Dk, int Dv, int page_size, int num_pages, int write_kv,
                                         cudaStream_t stream) {
  if (T == 0) return 0;
  DSP_REQUIRE(H > 0 && G > 0 && Dk > 0 && Dv > 0 && q_out, "dsp_qkv_conv_rotate_store: missing operand");
  const ConvIn p = {u, dtype, ld, 0, (H + G) * Dk + G * Dv, taps, w, hist, state_slot, q_start, seq_of_token, positions};
  if (const int rc = check(p, "dsp_qkv_conv_rotate_store")) return rc;
  DSP_REQUIRE(rot >= 0 && rot % 2 == 0 && rot <= Dk && (rot == 0 || inv_freq), "dsp_qkv_conv_rotate_store: rot=%d for keys of %d", rot, Dk);
  DSP_REQUIRE(!write_kv || (k_pool && v_pool && page_table && page_size > 0), "dsp_qkv_conv_rotate_store: no pools to write to");
  int* err = dsp_device_error_ptr();
  DSP_REQUIRE(err != nullptr, "dsp_qkv_conv_rotate_store: no device error word");
  const size_t smem = (size_t)(p.channels + rot) * sizeof(float);
  DSP_REQUIRE(smem <= 200 * 1024, "dsp_qkv_conv_rotate_store: rows of %d values do not fit shared memory", p.channels);
  static size_t configured = 48 * 1024;
  if (smem > configured) {
    DSP_CUDA(cudaFuncSetAttribute(qkv_conv_rotate_store_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    configured = smem;
  }
  DSP_CUDA(launch_plain(qkv_conv_rotate_store_kernel, dim3(T), dim3(256), smem, stream, p, page_table, pt_stride, k_pool,
                        v_pool, pool_dtype, inv_freq, rot, interleaved, head_norm, norm_eps, v_scale, q_out, ld_q, H, G, Dk,
                        Dv, page_size, num_pages, write_kv, err));
  DSP_CHECK_LAUNCH("dsp_qkv_conv_rotate_store");
  return 0;
}

extern "C" int dsp_conv_heads(const void* u, int dtype, long ld, int taps, const float* w, float* hist, const int* state_slot,
                              const int* q_start, const int* seq_of_token, const int* positions, int A, int B, int dim, int H,
                              int vdim, float eps, float a_scale, float* out, long ldo, int b_off, int a_off,
                              const float* step_bias, const float* a_log, float* steps, int T, cudaStream_t stream) {
  if (T == 0) return 0;
  DSP_REQUIRE(A >= 0 && B >= 0 && H > 0 && dim > 0 && vdim > 0, "dsp_conv_heads: %d and %d heads of %d, %d of %d", A, B, dim, H, vdim);
  const ConvIn p = {u, dtype, ld, 0, (A + B) * dim + H * vdim, taps, w, hist, state_slot, q_start, seq_of_token, positions};
  if (const int rc = check(p, "dsp_conv_heads")) return rc;
  DSP_REQUIRE(out && w && step_bias && a_log && steps, "dsp_conv_heads: missing operand");
  DSP_REQUIRE(A + B + H + 1 <= 65535, "dsp_conv_heads: too many heads");
  const int tok = T >= 256 ? 4 : 1, per = HEAD_WARPS * tok;
  DSP_CUDA(launch_plain(tok == 4 ? conv_heads_kernel<4> : conv_heads_kernel<1>, dim3((T + per - 1) / per, A + B + H + 1),
                        dim3(32 * HEAD_WARPS), 0, stream, p, T, A, B, dim, vdim, eps, a_scale, out, ldo, b_off, a_off, H, step_bias,
                        a_log, steps));
  DSP_CHECK_LAUNCH("dsp_conv_heads");
  return 0;
}
