// A recurrent mixer with a matrix memory per head: an exponential input gate, a forget gate, a running maximum that keeps
// both in range, and a normaliser (the matrix memory of xLSTM).
//
// Per head and token, with log gates i = cap tanh((zi + bi) / cap) and f = logsigmoid(cap tanh((zf + bf) / cap)) out of two
// logits, and m, S [dk][dv], n [dk] carried from token to token (32-bit, all zero at a request's start):
//   m' = max(f + m, i);  keep = exp(f + m - m');  put = exp(i - m')
//   S <- keep S + put k v^T;   n <- keep n + put k
//   o = S^T q / (max(|n . q|, exp(-m')) + 1e-6),  q including its factor dk^(-1/2)
// then o is divided by its root mean square over dv, multiplied by a weight per number and by sigmoid(gate).
//
// Kernels. `mlstm_gates` (a block per request and head): m' is a scan under the associative rule (F, I) o (F', I') =
// (F + F', max(I + F', I')), so a block takes as many tokens at a time as it has threads; it leaves keep, put and exp(-m')
// per token and moves m on. Only the differences of neighbouring m enter S and n, and they are formed from the m that are
// kept, so the scan's order of additions cannot disturb them. `mlstm_recurrence`: the columns of S are independent, n is one
// more column (its v is 1), so a group of lanes owns a column and walks the request's tokens. `mlstm_output` (a warp per
// token and head): denominator, norm, gate. In a step of single tokens the recurrence and the output kernel work the gates
// out themselves (the output kernel, which runs last, moves m on) and `mlstm_gates` is not launched.
#include <type_traits>

#include "common.cuh"

namespace {

struct Gates {
  float i, f;  // log input gate, log forget gate
};

__device__ __forceinline__ Gates log_gates(float zi, float zf, float bi, float bf, float cap) {
  Gates g;
  g.i = cap * tanhf((zi + bi) / cap);
  const float x = cap * tanhf((zf + bf) / cap);
  g.f = fminf(x, 0.f) - log1pf(expf(-fabsf(x)));
  return g;
}

// Rows of `proj` are `ld` numbers apart; the logits of head h sit at columns i_at + h and f_at + h.
struct MemoryParams {
  const float* proj;
  int ld, q_at, k_at, v_at, g_at, i_at, f_at;
  const float* i_bias;  // [heads]
  const float* f_bias;
  float cap;
  const int* seq_q_start;
  const int* seq_q_len;
  const int* seq_slot;
  int heads, dk, dv;
  float* S;     // [slots][heads][dk][dv]
  float* n;     // [slots][heads][dk]
  float* m;     // [slots][heads]
  float* keep;  // [tokens][heads], as are put and floor_
  float* put;
  float* floor_;
  float* num;   // [tokens][heads][dv]: S^T q
  float* den;   // [tokens][heads]: n . q
};

constexpr int kScanThreads = 256;

__global__ void __launch_bounds__(kScanThreads) mlstm_gates_kernel(const MemoryParams p) {
  __shared__ float warp_f[kScanThreads / 32], warp_i[kScanThreads / 32], m_row[kScanThreads + 1];
  let_successor_start();
  const int seq = blockIdx.x, head = blockIdx.y;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int start = p.seq_q_start[seq], len = p.seq_q_len[seq];
  float* slot = p.m + static_cast<int64_t>(p.seq_slot[seq]) * p.heads + head;
  const float bi = p.i_bias[head], bf = p.f_bias[head];
  wait_for_predecessor();
  float carried = *slot;
  for (int t0 = 0; t0 < len; t0 += blockDim.x) {
    const int t = t0 + tid;
    const int64_t at = static_cast<int64_t>(start + t);
    Gates g{-INFINITY, 0.f};  // past the end: the rule's neutral element
    if (t < len) g = log_gates(p.proj[at * p.ld + p.i_at + head], p.proj[at * p.ld + p.f_at + head], bi, bf, p.cap);
    float F = g.f, I = g.i;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float Fb = __shfl_up_sync(0xffffffffu, F, o), Ib = __shfl_up_sync(0xffffffffu, I, o);
      if (lane >= o) {
        I = fmaxf(Ib + F, I);
        F = Fb + F;
      }
    }
    if (lane == 31) warp_f[warp] = F, warp_i[warp] = I;
    __syncthreads();
    // What the warps in front of this one add up to, applied to the value carried in.
    float base = carried;
    for (int w = 0; w < warp; ++w) base = fmaxf(base + warp_f[w], warp_i[w]);
    const float m_new = fmaxf(base + F, I);
    m_row[tid + 1] = m_new;
    if (tid == 0) m_row[0] = carried;
    __syncthreads();
    if (t < len) {
      const float before = m_row[tid];
      p.keep[at * p.heads + head] = expf(g.f + before - m_new);
      p.put[at * p.heads + head] = expf(g.i - m_new);
      p.floor_[at * p.heads + head] = expf(-m_new);
    }
    carried = m_row[min(static_cast<int>(blockDim.x), len - t0)];
    __syncthreads();
  }
  if (tid == 0 && len > 0) *slot = carried;
}

constexpr int kRecurrenceThreads = 128;
constexpr int kStage = 8;

template <int kBytes>
__device__ __forceinline__ void stage_copy(float* smem, const float* gmem, bool valid) {
  const uint32_t s = static_cast<uint32_t>(__cvta_generic_to_shared(smem));
  const int bytes = valid ? kBytes : 0;
  asm volatile("cp.async.ca.shared.global [%0], [%1], %2, %3;" ::"r"(s), "l"(gmem), "n"(kBytes), "r"(bytes) : "memory");
}

// A column's dk rows are spread over LANES neighbouring lanes, PER rows each in registers: lane `part` holds rows
// (4 part .. 4 part + 3) + 4 LANES j, so that it reads q and k with 16-byte loads. The tokens' q, k, v, keep and put arrive
// kStage at a time by cp.async in a ring of two stages. The sums over lanes of a whole stage are formed together: at each
// exchange a lane gives away half of the tokens it still holds sums for and keeps the other half.
template <int PER, int LANES, bool SINGLE>
__global__ void __launch_bounds__(kRecurrenceThreads) mlstm_recurrence_kernel(const MemoryParams p, const int vec) {
  extern __shared__ __align__(16) float stage[];
  let_successor_start();
  constexpr int cols = kRecurrenceThreads / LANES;
  constexpr int padded = PER * LANES;
  constexpr int per_stage = kStage * (2 * padded + cols) + 2 * kStage;
  const int seq = blockIdx.x, head = blockIdx.y, col0 = blockIdx.z * cols;
  const int tid = threadIdx.x, part = tid % LANES, mine = tid / LANES, col = col0 + mine;
  const int start = p.seq_q_start[seq], len = p.seq_q_len[seq];
  const int64_t slot_head = static_cast<int64_t>(p.seq_slot[seq]) * p.heads + head;
  const bool live = col <= p.dv, is_n = col == p.dv;
  // Row r of this column of the state.
  float* column = is_n ? p.n + slot_head * p.dk : p.S + slot_head * p.dk * p.dv + col;
  const int64_t pitch = is_n ? 1 : p.dv;
  const float q_scale = 1.f / sqrtf(static_cast<float>(p.dk));
  auto row_of = [&](int i) { return (i >> 2) * 4 * LANES + part * 4 + (i & 3); };
  wait_for_predecessor();
  float s[PER];
#pragma unroll
  for (int i = 0; i < PER; ++i) s[i] = live && row_of(i) < p.dk ? column[row_of(i) * pitch] : 0.f;

  if constexpr (SINGLE) {
    const float* row = p.proj + static_cast<int64_t>(start) * p.ld;
    const Gates g = log_gates(row[p.i_at + head], row[p.f_at + head], p.i_bias[head], p.f_bias[head], p.cap);
    const float before = p.m[slot_head];
    const float m_new = fmaxf(g.f + before, g.i);
    const float keep = expf(g.f + before - m_new);
    const float put = expf(g.i - m_new) * (is_n || !live ? 1.f : row[p.v_at + head * p.dv + col]);
    float sum = 0.f;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      const int r = row_of(i);
      if (r < p.dk) {
        s[i] = fmaf(row[p.k_at + head * p.dk + r], put, keep * s[i]);
        sum = fmaf(row[p.q_at + head * p.dk + r], s[i], sum);
      }
    }
#pragma unroll
    for (int o = LANES >> 1; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    if (live && part == 0) {
      const int64_t at = static_cast<int64_t>(start) * p.heads + head;
      if (is_n) p.den[at] = sum * q_scale;
      else p.num[at * p.dv + col] = sum * q_scale;
    }
  } else {
    auto fetch = [&](int buffer, int t0) {
      float* sq = stage + buffer * per_stage;
      float* sk = sq + kStage * padded;
      float* sv = sk + kStage * padded;
      float* sg = sv + kStage * cols;
      const int count = min(kStage, len - t0);
      const float* first = p.proj + static_cast<int64_t>(start + t0) * p.ld;
      if (vec) {
        for (int idx = tid * 4; idx < count * padded; idx += kRecurrenceThreads * 4) {
          const int j = idx / padded, row = idx % padded;
          const float* at = first + static_cast<int64_t>(j) * p.ld + head * p.dk + (row < p.dk ? row : 0);
          stage_copy<16>(sq + idx, at + p.q_at, row < p.dk);
          stage_copy<16>(sk + idx, at + p.k_at, row < p.dk);
        }
        if constexpr (cols >= 4) {
          for (int idx = tid * 4; idx < count * cols; idx += kRecurrenceThreads * 4) {
            const int j = idx / cols, c = col0 + idx % cols;
            stage_copy<16>(sv + idx, first + static_cast<int64_t>(j) * p.ld + p.v_at + head * p.dv + (c < p.dv ? c : 0), c < p.dv);
          }
        }
      } else {
        for (int idx = tid; idx < count * padded; idx += kRecurrenceThreads) {
          const int j = idx / padded, row = idx % padded;
          const float* at = first + static_cast<int64_t>(j) * p.ld + head * p.dk + (row < p.dk ? row : 0);
          stage_copy<4>(sq + idx, at + p.q_at, row < p.dk);
          stage_copy<4>(sk + idx, at + p.k_at, row < p.dk);
        }
      }
      if (!vec || cols < 4) {
        for (int idx = tid; idx < count * cols; idx += kRecurrenceThreads) {
          const int j = idx / cols, c = col0 + idx % cols;
          stage_copy<4>(sv + idx, first + static_cast<int64_t>(j) * p.ld + p.v_at + head * p.dv + (c < p.dv ? c : 0), c < p.dv);
        }
      }
      if (tid < count) {
        const int64_t at = static_cast<int64_t>(start + t0 + tid) * p.heads + head;
        stage_copy<4>(sg + tid, p.keep + at, true);
        stage_copy<4>(sg + kStage + tid, p.put + at, true);
      }
    };
    if (len > 0) fetch(0, 0);
    asm volatile("cp.async.commit_group;" ::: "memory");
    for (int t0 = 0, buffer = 0; t0 < len; t0 += kStage, buffer ^= 1) {
      if (t0 + kStage < len) fetch(buffer ^ 1, t0 + kStage);
      asm volatile("cp.async.commit_group;" ::: "memory");
      asm volatile("cp.async.wait_group 1;" ::: "memory");
      __syncthreads();
      const float* sq = stage + buffer * per_stage;
      const float* sk = sq + kStage * padded;
      const float* sv = sk + kStage * padded;
      const float* sg = sv + kStage * cols;
      const int count = min(kStage, len - t0);
      float sums[kStage];
      auto token = [&](int j) {
        const float keep = sg[j];
        const float put = sg[kStage + j] * (is_n ? 1.f : sv[j * cols + mine]);
        float a = 0.f, b = 0.f;
#pragma unroll
        for (int c = 0; c < PER / 4; ++c) {
          const float4 k4 = *reinterpret_cast<const float4*>(sk + j * padded + c * 4 * LANES + part * 4);
          const float4 q4 = *reinterpret_cast<const float4*>(sq + j * padded + c * 4 * LANES + part * 4);
          s[4 * c] = fmaf(k4.x, put, keep * s[4 * c]);
          s[4 * c + 1] = fmaf(k4.y, put, keep * s[4 * c + 1]);
          s[4 * c + 2] = fmaf(k4.z, put, keep * s[4 * c + 2]);
          s[4 * c + 3] = fmaf(k4.w, put, keep * s[4 * c + 3]);
          a = fmaf(q4.x, s[4 * c], a), b = fmaf(q4.y, s[4 * c + 1], b);
          a = fmaf(q4.z, s[4 * c + 2], a), b = fmaf(q4.w, s[4 * c + 3], b);
        }
        sums[j] = a + b;
      };
      if (count == kStage) {
#pragma unroll
        for (int j = 0; j < kStage; ++j) token(j);
      } else {
#pragma unroll
        for (int j = 0; j < kStage; ++j) {
          sums[j] = 0.f;
          if (j < count) token(j);
        }
      }
      // Halve the tokens a lane answers for with every exchange; when one is left, plain sums over what lanes remain.
      int first = 0, held = kStage;
#pragma unroll
      for (int o = LANES >> 1; o > 0; o >>= 1) {
        if (held > 1) {
          held >>= 1;
          const bool upper = (part & o) != 0;
#pragma unroll
          for (int j = 0; j < kStage / 2; ++j)
            if (j < held) {
              const float give = upper ? sums[j] : sums[j + held], take = upper ? sums[j + held] : sums[j];
              sums[j] = take + __shfl_xor_sync(0xffffffffu, give, o);
            }
          if (upper) first += held;
        } else {
          sums[0] += __shfl_xor_sync(0xffffffffu, sums[0], o);
        }
      }
      constexpr int kSharers = LANES > kStage ? LANES / kStage : 1;  // lanes that end with the same token's sum
      if (live && part % kSharers == 0) {
#pragma unroll
        for (int j = 0; j < kStage; ++j) {
          if (j >= held || first + j >= count) continue;
          const int64_t at = static_cast<int64_t>(start + t0 + first + j) * p.heads + head;
          if (is_n) p.den[at] = sums[j] * q_scale;
          else p.num[at * p.dv + col] = sums[j] * q_scale;
        }
      }
      __syncthreads();
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
  }
#pragma unroll
  for (int i = 0; i < PER; ++i)
    if (live && row_of(i) < p.dk) column[row_of(i) * pitch] = s[i];
}

// One warp per (token, head). SINGLE: the token is its request's only one; exp(-m') is worked out here and m moves on.
template <typename T, bool SINGLE>
__global__ void mlstm_output_kernel(const MemoryParams p, const float* __restrict__ weight, float eps, int rows, T* out) {
  let_successor_start();
  const int lane = threadIdx.x & 31;
  const int64_t item = static_cast<int64_t>(blockIdx.x) * (blockDim.x >> 5) + (threadIdx.x >> 5);
  wait_for_predecessor();
  if (item >= static_cast<int64_t>(rows) * p.heads) return;
  const int head = static_cast<int>(item % p.heads);
  const int64_t t = item / p.heads;
  const float* row = p.proj + t * p.ld;
  float least;
  if constexpr (SINGLE) {  // requests and tokens coincide, in the same order
    float* slot = p.m + static_cast<int64_t>(p.seq_slot[t]) * p.heads + head;
    const Gates g = log_gates(row[p.i_at + head], row[p.f_at + head], p.i_bias[head], p.f_bias[head], p.cap);
    const float m_new = fmaxf(g.f + *slot, g.i);
    least = expf(-m_new);
    __syncwarp();
    if (lane == 0) *slot = m_new;
  } else {
    least = p.floor_[item];
  }
  const float* num = p.num + item * p.dv;
  const float inv_den = 1.f / (fmaxf(fabsf(p.den[item]), least) + 1e-6f);
  float ss = 0.f;
  for (int i = lane; i < p.dv; i += 32) {
    const float o = num[i] * inv_den;
    ss = fmaf(o, o, ss);
  }
  ss = warp_sum(ss);
  const float inv = inv_den / sqrtf(ss / static_cast<float>(p.dv) + eps);
  for (int i = lane; i < p.dv; i += 32) {
    const float gate = 1.f / (1.f + expf(-row[p.g_at + head * p.dv + i]));
    out[item * p.dv + i] = from_f32<T>(num[i] * inv * weight[head * p.dv + i] * gate);
  }
}

}  // namespace

// The whole of the mixer between its two products. `proj` (float, rows `ld` apart) holds q, k (heads * dk each), v and the
// gate logits (heads * dv each) and the two gates' logits (heads each) from the columns given. `single`: every request of the
// step feeds one token (two launches instead of three). `norm`: [heads * dv]; `out`: [tokens][heads * dv].
B200_API int b200_mlstm(const float* proj, int ld, int q_at, int k_at, int v_at, int g_at, int i_at, int f_at, const float* i_bias,
                        const float* f_bias, float cap, const int* seq_q_start, const int* seq_q_len, const int* seq_slot, int seqs,
                        int tokens, int single, int heads, int dk, int dv, float* S, float* n, float* m, float* keep, float* put,
                        float* least, float* num, float* den, const float* norm, float eps, void* out, int dtype, cudaStream_t stream) {
  if (tokens == 0 || seqs == 0) return 0;
  B200_REQUIRE(tokens > 0 && seqs > 0 && heads > 0 && heads <= 65535 && dk > 0 && dv > 0 && cap > 0.f, "mlstm: bad sizes");
  B200_REQUIRE(dk <= 1024, "mlstm: %d key channels per head, at most 1024", dk);
  B200_REQUIRE(!single || tokens == seqs, "mlstm: a step of single tokens has as many tokens as requests");
  B200_REQUIRE(single || (keep != nullptr && put != nullptr && least != nullptr), "mlstm: no room for the gates");
  MemoryParams p{proj, ld, q_at, k_at, v_at, g_at, i_at, f_at, i_bias, f_bias, cap, seq_q_start, seq_q_len, seq_slot,
                 heads, dk, dv, S, n, m, keep, put, least, num, den};
  if (!single) {
    launch_kernel(mlstm_gates_kernel, dim3(seqs, heads), dim3(kScanThreads), 0, stream, p);
    if (int status = b200_check_launch("mlstm_gates")) return status;
  }
  int lanes = 1;
  while ((dk + lanes - 1) / lanes > 8 && lanes < 32) lanes *= 2;
  const int rows = (dk + lanes - 1) / lanes;
  const int per = rows <= 8 ? 8 : (rows <= 16 ? 16 : 32);
  const int cols = kRecurrenceThreads / lanes;
  const dim3 grid(seqs, heads, (dv + 1 + cols - 1) / cols);
  B200_REQUIRE(grid.z <= 65535, "mlstm: too many columns");
  const size_t smem = single ? 0 : sizeof(float) * 2 * (kStage * (2 * per * lanes + cols) + 2 * kStage);
  B200_REQUIRE(smem <= 200 * 1024, "mlstm: the staged tokens do not fit shared memory");
  const bool aligned = reinterpret_cast<uintptr_t>(proj) % 16 == 0;
  const int vec = aligned && dk % 4 == 0 && dv % 4 == 0 && ld % 4 == 0 && q_at % 4 == 0 && k_at % 4 == 0 && v_at % 4 == 0 ? 1 : 0;
  auto launch = [&](auto kernel) {
    if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    launch_kernel(kernel, grid, dim3(kRecurrenceThreads), smem, stream, p, vec);
  };
  auto by_shape = [&](auto one) {
    constexpr bool kSingle = decltype(one)::value;
    if (per == 32) launch(mlstm_recurrence_kernel<32, 32, kSingle>);
    else if (per == 16) launch(mlstm_recurrence_kernel<16, 32, kSingle>);
    else if (lanes == 32) launch(mlstm_recurrence_kernel<8, 32, kSingle>);
    else if (lanes == 16) launch(mlstm_recurrence_kernel<8, 16, kSingle>);
    else if (lanes == 8) launch(mlstm_recurrence_kernel<8, 8, kSingle>);
    else if (lanes == 4) launch(mlstm_recurrence_kernel<8, 4, kSingle>);
    else if (lanes == 2) launch(mlstm_recurrence_kernel<8, 2, kSingle>);
    else launch(mlstm_recurrence_kernel<8, 1, kSingle>);
  };
  if (single) by_shape(std::true_type{});
  else by_shape(std::false_type{});
  if (int status = b200_check_launch("mlstm_recurrence")) return status;
  const int threads = 128;
  const unsigned blocks = static_cast<unsigned>((static_cast<int64_t>(tokens) * heads + 3) / 4);
  auto output = [&](auto kernel, auto* typed) { launch_kernel(kernel, dim3(blocks), dim3(threads), 0, stream, p, norm, eps, tokens, typed); };
  if (dtype == DTYPE_F32) {
    if (single) output(mlstm_output_kernel<float, true>, static_cast<float*>(out));
    else output(mlstm_output_kernel<float, false>, static_cast<float*>(out));
  } else if (dtype == DTYPE_BF16) {
    if (single) output(mlstm_output_kernel<__nv_bfloat16, true>, static_cast<__nv_bfloat16*>(out));
    else output(mlstm_output_kernel<__nv_bfloat16, false>, static_cast<__nv_bfloat16*>(out));
  } else {
    return b200_fail("mlstm: unknown dtype %d", dtype);
  }
  return b200_check_launch("mlstm_output");
}
