// The gated delta rule with one decay per head: the recurrence over prompt portions and the whole mixer of decoded tokens.
//
// Per head, with a state S [dk][dv] (32-bit, zero at a request's start) carried from token to token:
//   S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q   (the read-out sees the token's own write).
// With one factor g for the whole state both products can read the state as the token before left it,
//   u = beta (v - g (S^T k)),  o = g (S^T q) + (k . q) u,  S <- g S + k u^T,
// so that a token's two sums over key channels depend on nothing but the old state and are added up together.
//
// `delta_head_recurrence`: the columns of S are independent; a group of lanes owns a column and walks the request's tokens
// (q, k, v, beta, log g and k . q as `delta_prepare` in delta_rule.cu leaves them).
// `delta_head_step` (steps in which every request feeds one token): short convolution and its state, unit vectors, beta,
// decay, recurrence, norm of the head's output and its gate in one kernel, one block per request and head. The state and
// the convolution's history were left by an earlier step, so a block reads them before it waits for the projection in front.
#include <type_traits>

#include "common.cuh"

namespace {

__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float softplus_f(float x) { return x > 20.f ? x : log1pf(expf(x)); }

// A block owns `cols` columns of one head of one request; a column's dk rows are spread over `LANES` neighbouring lanes, PER
// neighbouring rows per lane in registers. A lane reads four neighbouring numbers of q and k with one 16-byte load; in shared
// memory a lane's rows are followed by four unused numbers, which puts the lanes that load together on different banks. The
// tokens arrive kStage at a time by cp.async in a ring of two stages, so the next ones load while these are worked on.
constexpr int kRecurrenceThreads = 128;
constexpr int kStage = 8;

template <int kBytes>
__device__ __forceinline__ void stage_copy(float* smem, const float* gmem, bool valid) {
  const uint32_t s = static_cast<uint32_t>(__cvta_generic_to_shared(smem));
  const int bytes = valid ? kBytes : 0;
  asm volatile("cp.async.ca.shared.global [%0], [%1], %2, %3;" ::"r"(s), "l"(gmem), "n"(kBytes), "r"(bytes) : "memory");
}

template <int PER, int LANES>
__global__ void __launch_bounds__(kRecurrenceThreads)
delta_head_recurrence_kernel(const float* q, const float* k, const float* v, const float* beta, const float* log_decay, const float* kq,
                             const int* seq_q_start, const int* seq_q_len, const int* seq_slot, int heads, int kv_heads, int dk, int dv, int vec,
                             float* state, float* out) {
  extern __shared__ __align__(16) float stage[];
  let_successor_start();
  constexpr int cols = kRecurrenceThreads / LANES;
  constexpr int lane_span = PER + 4;
  constexpr int padded = lane_span * LANES;
  constexpr int per_stage = kStage * (2 * padded + cols + 4);
  const int seq = blockIdx.x, head = blockIdx.y, col0 = blockIdx.z * cols;
  const int tid = threadIdx.x;
  const int part = tid % LANES, col = col0 + tid / LANES;
  const int start = seq_q_start[seq], len = seq_q_len[seq];
  const int kvh = head / (heads / kv_heads);
  const bool live = col < dv;
  float* s_base = state + (static_cast<int64_t>(seq_slot[seq]) * heads + head) * dk * dv;
  wait_for_predecessor();
  // Rows past dk (when dk is no multiple of the lanes) hold zeros in q and k and stay zero.
  auto fetch = [&](int buffer, int t0) {
    float* sq = stage + buffer * per_stage;
    float* sk = sq + kStage * padded;
    float* sv = sk + kStage * padded;
    float* sc = sv + kStage * cols;  // per token: beta, log decay, k . q, unused
    const int count = min(kStage, len - t0);
    const int64_t first = static_cast<int64_t>(start) + t0;
    auto vectors = [&](auto width) {
      constexpr int W = decltype(width)::value;
      for (int idx = tid * W; idx < count * padded; idx += kRecurrenceThreads * W) {
        const int j = idx / padded, place = idx % padded;
        if (place % lane_span >= PER) continue;
        const int row = place / lane_span * PER + place % lane_span;
        const int64_t at = ((first + j) * kv_heads + kvh) * dk + (row < dk ? row : 0);
        stage_copy<4 * W>(sq + idx, q + at, row < dk);
        stage_copy<4 * W>(sk + idx, k + at, row < dk);
      }
      for (int idx = tid * W; idx < count * cols; idx += kRecurrenceThreads * W) {
        const int j = idx / cols, c = col0 + idx % cols;
        stage_copy<4 * W>(sv + idx, v + ((first + j) * heads + head) * dv + (c < dv ? c : 0), c < dv);
      }
    };
    if (vec) vectors(std::integral_constant<int, 4>{});
    else vectors(std::integral_constant<int, 1>{});
    if (tid < 3 * kStage) {
      const int j = tid / 3, n = tid % 3;
      if (j < count) {
        const float* from = n == 0 ? beta + (first + j) * heads + head : (n == 1 ? log_decay + (first + j) * heads + head : kq + (first + j) * kv_heads + kvh);
        stage_copy<4>(sc + j * 4 + n, from, true);
      }
    }
  };
  float s[PER];
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int row = part * PER + i;
    s[i] = (live && row < dk) ? s_base[static_cast<int64_t>(row) * dv + col] : 0.f;
  }
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
    const float* sc = sv + kStage * cols;
    const int count = min(kStage, len - t0);
    auto token = [&](int j) {
      const int at = j * padded + part * lane_span;
      const float4 c = *reinterpret_cast<const float4*>(sc + j * 4);
      const float g = expf(c.y);
      const float vc = sv[j * cols + tid / LANES];
      float qv[PER], kv[PER];
#pragma unroll
      for (int i = 0; i < PER; i += 4) {
        *reinterpret_cast<float4*>(qv + i) = *reinterpret_cast<const float4*>(sq + at + i);
        *reinterpret_cast<float4*>(kv + i) = *reinterpret_cast<const float4*>(sk + at + i);
      }
      float k0 = 0.f, k1 = 0.f, q0 = 0.f, q1 = 0.f;
#pragma unroll
      for (int i = 0; i < PER; i += 2) {
        k0 = fmaf(kv[i], s[i], k0), k1 = fmaf(kv[i + 1], s[i + 1], k1);
        q0 = fmaf(qv[i], s[i], q0), q1 = fmaf(qv[i + 1], s[i + 1], q1);
      }
      float ks = k0 + k1, qs = q0 + q1;
#pragma unroll
      for (int o = LANES >> 1; o > 0; o >>= 1) {
        const float from_k = __shfl_xor_sync(0xffffffffu, ks, o), from_q = __shfl_xor_sync(0xffffffffu, qs, o);
        ks += from_k, qs += from_q;
      }
      const float u = c.x * fmaf(-g, ks, vc);
#pragma unroll
      for (int i = 0; i < PER; ++i) s[i] = fmaf(kv[i], u, g * s[i]);
      if (live && part == 0) out[(static_cast<int64_t>(start) + t0 + j) * heads * dv + head * dv + col] = fmaf(c.z, u, g * qs);
    };
    if (count == kStage) {  // a full stage is unrolled: the next token's operands load beside this one's sums
#pragma unroll
      for (int j = 0; j < kStage; ++j) token(j);
    } else {
      for (int j = 0; j < count; ++j) token(j);
    }
    __syncthreads();
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int row = part * PER + i;
    if (live && row < dk) s_base[static_cast<int64_t>(row) * dv + col] = s[i];
  }
}

// ---- the whole mixer of decoded tokens ----------------------------------------------------------------------------------

// Row of `proj`: [q (kv_heads*dk) | k (kv_heads*dk) | v (heads*dv) | b (heads) | a (heads) | gate (heads*dv)].
struct StepShape {
  int ld, heads, kv_heads, dk, dv, taps;
  int slices;       // warps that share a column of S: the block's warps / column tiles
  int slice_rows;   // rows of S per slice, at most PER
  float eps;
};

constexpr int kStepThreads = 512;
constexpr int kStepWarps = kStepThreads / 32;

// A warp holds 32 neighbouring columns of `slice_rows` rows of S, a row's 32 numbers in one access. The heads that share a
// q/k head are one thread-block cluster (its first block moves their convolution history on, once all have read it).
template <typename T, int PER>
__global__ void __launch_bounds__(kStepThreads, PER <= 32 ? 2 : 1)
delta_head_step_kernel(const T* proj, const float* __restrict__ taps_w, T* conv_state, const float* __restrict__ a_log,
                       const float* __restrict__ dt_bias, const float* __restrict__ norm_weight, const int* __restrict__ seq_q_start,
                       const int* __restrict__ seq_slot, const StepShape p, float* state, T* out) {
  extern __shared__ __align__(16) float step_smem[];
  let_successor_start();
  const int group = p.heads / p.kv_heads;
  const int head = blockIdx.x, kvh = head / group, seq = blockIdx.y;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int dk = p.dk, dv = p.dv, dk_pad = (dk + 3) & ~3;
  const int channels = 2 * p.kv_heads * dk + p.heads * dv;
  const int mine = 2 * dk + dv;  // this block's channels: q and k of the shared head, v of its own
  float* qs = step_smem;                // [dk_pad] q, then k, as rows of the projection become them
  float* ks = qs + dk_pad;
  float* vs = ks + dk_pad;              // [dv]
  float* sums = vs + dv;                // [2][slices][dv]: partial S^T k and S^T q
  float* ss = sums + 2 * p.slices * dv; // [kStepWarps]
  const int slot = seq_slot[seq];
  const int t = seq_q_start[seq];
  T* history = conv_state + static_cast<int64_t>(slot) * (p.taps - 1) * channels;
  auto channel_of = [&](int c) {  // of the projection's convolved columns
    return c < dk ? kvh * dk + c : (c < 2 * dk ? p.kv_heads * dk + kvh * dk + c - dk : 2 * p.kv_heads * dk + head * dv + c - 2 * dk);
  };

  // What earlier steps left: this warp's part of S, and the convolution over its history.
  const int tiles = (dv + 31) / 32;
  const int slice = warp / tiles, col = (warp % tiles) * 32 + lane;
  const int row0 = slice * p.slice_rows;
  const int rows = slice < p.slices ? min(p.slice_rows, dk - row0) : 0;  // may be negative past the last row
  const bool live = slice < p.slices && col < dv;
  float* s_base = state + (static_cast<int64_t>(slot) * p.heads + head) * dk * dv + static_cast<int64_t>(row0) * dv + col;
  float s[PER];
#pragma unroll
  for (int i = 0; i < PER; ++i) s[i] = (live && i < rows) ? s_base[static_cast<int64_t>(i) * dv] : 0.f;
  for (int c = tid; c < mine; c += kStepThreads) {
    const int ch = channel_of(c);
    float acc = 0.f;
    for (int j = 0; j + 1 < p.taps; ++j) acc = fmaf(taps_w[ch * p.taps + j], to_f32<T>(history[static_cast<int64_t>(j) * channels + ch]), acc);
    (c < dk ? qs + c : (c < 2 * dk ? ks + c - dk : vs + c - 2 * dk))[0] = acc;
  }
  if (tid < dk_pad - dk) qs[dk + tid] = ks[dk + tid] = 0.f;
  const float rate = -expf(a_log[head]), bias = dt_bias[head];
  if (group > 1) asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");  // this block has read the shared history
  wait_for_predecessor();

  const T* row = proj + static_cast<int64_t>(t) * p.ld;
  for (int c = tid; c < mine; c += kStepThreads) {
    const int ch = channel_of(c);
    float* y = c < dk ? qs + c : (c < 2 * dk ? ks + c - dk : vs + c - 2 * dk);
    const float acc = fmaf(taps_w[ch * p.taps + p.taps - 1], to_f32<T>(row[ch]), *y);
    *y = acc * sigmoid_f(acc);
  }
  const float beta = sigmoid_f(to_f32<T>(row[channels + head]));
  const float g = expf(rate * softplus_f(to_f32<T>(row[channels + p.heads + head]) + bias));
  __syncthreads();
  // Lengths of q and k and their product, worked out by every warp for itself; S^T k and S^T q over this slice's rows of the
  // old state. The lengths are factors of the finished sums.
  float ss_q = 0.f, ss_k = 0.f, dot = 0.f;
  for (int i = lane; i < dk; i += 32) {
    const float a = qs[i], b = ks[i];
    ss_q = fmaf(a, a, ss_q), ss_k = fmaf(b, b, ss_k), dot = fmaf(a, b, dot);
  }
  ss_q = warp_sum(ss_q), ss_k = warp_sum(ss_k), dot = warp_sum(dot);
  const float inv_q = (1.f / sqrtf(ss_q + 1e-6f)) * (1.f / sqrtf(static_cast<float>(dk))), inv_k = 1.f / sqrtf(ss_k + 1e-6f);
  float k0 = 0.f, k1 = 0.f, q0 = 0.f, q1 = 0.f;
#pragma unroll
  for (int i = 0; i < PER; i += 2) {
    if (i < rows) {
      k0 = fmaf(ks[row0 + i], s[i], k0), q0 = fmaf(qs[row0 + i], s[i], q0);
      if (i + 1 < rows) k1 = fmaf(ks[row0 + i + 1], s[i + 1], k1), q1 = fmaf(qs[row0 + i + 1], s[i + 1], q1);
    }
  }
  if (live) {
    sums[slice * dv + col] = k0 + k1;
    sums[(p.slices + slice) * dv + col] = q0 + q1;
  }
  __syncthreads();
  float o = 0.f;
  if (live) {
    float sk = 0.f, sq = 0.f;
    for (int j = 0; j < p.slices; ++j) sk += sums[j * dv + col], sq += sums[(p.slices + j) * dv + col];
    const float u = beta * fmaf(-g, sk * inv_k, vs[col]);
    o = fmaf(dot * inv_k * inv_q, u, g * (sq * inv_q));
    const float ku = inv_k * u;
#pragma unroll
    for (int i = 0; i < PER; ++i)
      if (i < rows) s_base[static_cast<int64_t>(i) * dv] = fmaf(ks[row0 + i], ku, g * s[i]);
  }
  // Norm over the head's columns and the gate; the first slice's warps hold every column once.
  const bool writer = live && slice == 0;
  const float own = warp_sum(writer ? o * o : 0.f);
  if (lane == 0) ss[warp] = own;
  // The convolution's history moves on by this token: v's channels are this block's alone, q's and k's the cluster's.
  for (int c = 2 * dk + tid; c < mine; c += kStepThreads) {
    const int ch = channel_of(c);
    for (int j = 0; j + 2 < p.taps; ++j) history[static_cast<int64_t>(j) * channels + ch] = history[static_cast<int64_t>(j + 1) * channels + ch];
    if (p.taps > 1) history[static_cast<int64_t>(p.taps - 2) * channels + ch] = row[ch];
  }
  __syncthreads();
  if (writer) {
    float total = 0.f;
    for (int w = 0; w < tiles; ++w) total += ss[w];
    const float inv = 1.f / sqrtf(total / static_cast<float>(dv) + p.eps);
    const float x = to_f32<T>(row[channels + 2 * p.heads + head * dv + col]);
    out[(static_cast<int64_t>(t) * p.heads + head) * dv + col] = from_f32<T>(o * inv * norm_weight[col] * (x * sigmoid_f(x)));
  }
  if (group > 1) asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
  if (head % group == 0) {
    for (int c = tid; c < 2 * dk; c += kStepThreads) {
      const int ch = channel_of(c);
      for (int j = 0; j + 2 < p.taps; ++j) history[static_cast<int64_t>(j) * channels + ch] = history[static_cast<int64_t>(j + 1) * channels + ch];
      if (p.taps > 1) history[static_cast<int64_t>(p.taps - 2) * channels + ch] = row[ch];
    }
  }
}

struct StepPlan {
  int slices, slice_rows;
  size_t smem;
};

constexpr int kStepMaxRows = 64;

// False when a head's state does not fit one block's registers or its heads one cluster.
bool plan_step(int heads, int kv_heads, int dk, int dv, StepPlan* plan) {
  const int tiles = (dv + 31) / 32;
  if (dk <= 0 || dv <= 0 || kv_heads <= 0 || heads % kv_heads || heads / kv_heads > 8 || tiles > kStepWarps) return false;
  plan->slices = kStepWarps / tiles;
  plan->slice_rows = (dk + plan->slices - 1) / plan->slices;
  plan->smem = sizeof(float) * (2 * ((dk + 3) & ~3) + dv + 2 * plan->slices * dv + kStepWarps);
  return plan->slice_rows <= kStepMaxRows && plan->smem <= 48 * 1024;
}

template <typename T, int PER>
cudaError_t launch_step(const StepPlan& plan, int seqs, cudaStream_t stream, const T* proj, const float* taps_w, T* conv_state, const float* a_log,
                        const float* dt_bias, const float* norm_weight, const int* seq_q_start, const int* seq_slot, const StepShape& shape,
                        float* state, T* out) {
  cudaLaunchConfig_t config = {};
  config.gridDim = dim3(shape.heads, seqs);
  config.blockDim = dim3(kStepThreads);
  config.dynamicSmemBytes = plan.smem;
  config.stream = stream;
  cudaLaunchAttribute attributes[2];
  int count = 0;
  const int group = shape.heads / shape.kv_heads;
  if (group > 1) {
    attributes[count].id = cudaLaunchAttributeClusterDimension;
    attributes[count].val.clusterDim.x = group;
    attributes[count].val.clusterDim.y = 1;
    attributes[count].val.clusterDim.z = 1;
    ++count;
  }
  if (b200_overlap_enabled()) {
    attributes[count].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attributes[count].val.programmaticStreamSerializationAllowed = 1;
    ++count;
  }
  config.attrs = attributes;
  config.numAttrs = count;
  return cudaLaunchKernelEx(&config, delta_head_step_kernel<T, PER>, proj, taps_w, conv_state, a_log, dt_bias, norm_weight, seq_q_start, seq_slot,
                            shape, state, out);
}

}  // namespace

B200_API int b200_delta_head_recurrence(const float* q, const float* k, const float* v, const float* beta, const float* log_decay, const float* kq,
                                        const int* seq_q_start, const int* seq_q_len, const int* seq_slot, int seqs, int max_q_len, int heads,
                                        int kv_heads, int dk, int dv, float* state, float* out, cudaStream_t stream) {
  if (seqs == 0) return 0;
  B200_REQUIRE(seqs > 0 && heads > 0 && heads <= 65535 && kv_heads > 0 && heads % kv_heads == 0 && dk > 0 && dv > 0,
               "delta_head_recurrence: bad sizes");
  B200_REQUIRE(dk <= 1024, "delta_head_recurrence: %d key channels per head, at most 1024", dk);
  // Lanes per column: enough that a lane holds at most 8 rows (up to 32 rows when even a whole warp
  // per column leaves more).
  int lanes = 1;
  while ((dk + lanes - 1) / lanes > 8 && lanes < 32) lanes *= 2;
  const int rows = (dk + lanes - 1) / lanes;
  const int per = rows <= 8 ? 8 : (rows <= 16 ? 16 : 32);
  const int cols = kRecurrenceThreads / lanes;
  const dim3 grid(seqs, heads, (dv + cols - 1) / cols);
  B200_REQUIRE(grid.z <= 65535, "delta_head_recurrence: too many columns");
  const size_t smem = sizeof(float) * 2 * kStage * (2 * (per + 4) * lanes + cols + 4);
  const auto aligned = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
  const int vec = dk % 4 == 0 && dv % 4 == 0 && cols % 4 == 0 && aligned(q) && aligned(k) && aligned(v) ? 1 : 0;
  // A step with prompt portions launches the ordinary way: made resident early, the few blocks are packed several to an SM
  // onto the SMs that the predecessor's last wave leaves free and walk their tokens there to the end.
  const bool ordered = max_q_len > kStage;
  auto launch = [&](auto kernel) {
    if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    launch_kernel_as(ordered, kernel, grid, dim3(kRecurrenceThreads), smem, stream, q, k, v, beta, log_decay, kq, seq_q_start, seq_q_len, seq_slot,
                     heads, kv_heads, dk, dv, vec, state, out);
  };
  if (per == 32) launch(delta_head_recurrence_kernel<32, 32>);
  else if (per == 16) launch(delta_head_recurrence_kernel<16, 32>);
  else if (lanes == 32) launch(delta_head_recurrence_kernel<8, 32>);
  else if (lanes == 16) launch(delta_head_recurrence_kernel<8, 16>);
  else if (lanes == 8) launch(delta_head_recurrence_kernel<8, 8>);
  else if (lanes == 4) launch(delta_head_recurrence_kernel<8, 4>);
  else if (lanes == 2) launch(delta_head_recurrence_kernel<8, 2>);
  else launch(delta_head_recurrence_kernel<8, 1>);
  return b200_check_launch("delta_head_recurrence");
}

// Whether `b200_delta_head_step` takes the shape; the caller runs prepare, recurrence and output otherwise.
B200_API int b200_delta_head_step_supported(int heads, int kv_heads, int dk, int dv) {
  StepPlan plan;
  return plan_step(heads, kv_heads, dk, dv, &plan) ? 1 : 0;
}

// One token of each of `seqs` requests.
B200_API int b200_delta_head_step(const void* proj, int ld, const float* taps_w, int taps, void* conv_state, const float* a_log, const float* dt_bias,
                                  const float* norm_weight, float eps, const int* seq_q_start, const int* seq_slot, int seqs, int heads, int kv_heads,
                                  int dk, int dv, float* state, void* out, int dtype, cudaStream_t stream) {
  if (seqs == 0) return 0;
  StepPlan plan;
  B200_REQUIRE(seqs > 0 && seqs <= 65535 && taps >= 1 && plan_step(heads, kv_heads, dk, dv, &plan), "delta_head_step: shape not taken");
  B200_REQUIRE(ld >= 2 * kv_heads * dk + 2 * heads * dv + 2 * heads, "delta_head_step: rows of %d numbers do not hold the projections", ld);
  const StepShape shape{ld, heads, kv_heads, dk, dv, taps, plan.slices, plan.slice_rows, eps};
  auto launch = [&](auto zero) -> cudaError_t {
    using T = decltype(zero);
    const T* in = static_cast<const T*>(proj);
    T* history = static_cast<T*>(conv_state);
    T* to = static_cast<T*>(out);
    if (plan.slice_rows <= 16) return launch_step<T, 16>(plan, seqs, stream, in, taps_w, history, a_log, dt_bias, norm_weight, seq_q_start, seq_slot, shape, state, to);
    if (plan.slice_rows <= 32) return launch_step<T, 32>(plan, seqs, stream, in, taps_w, history, a_log, dt_bias, norm_weight, seq_q_start, seq_slot, shape, state, to);
    return launch_step<T, 64>(plan, seqs, stream, in, taps_w, history, a_log, dt_bias, norm_weight, seq_q_start, seq_slot, shape, state, to);
  };
  cudaError_t status;
  if (dtype == DTYPE_F32) status = launch(float{});
  else if (dtype == DTYPE_BF16) status = launch(__nv_bfloat16{});
  else return b200_fail("delta_head_step: unknown dtype %d", dtype);
  if (status != cudaSuccess) return b200_fail("delta_head_step: %s", cudaGetErrorString(status));
  return b200_check_launch("delta_head_step");
}
