// The gated delta rule with one decay per head over prompt portions, 32 tokens at a time.
//
// Token by token (delta_head.cu) a portion costs tokens x the latency of one step, however few columns a head has. Over a chunk
// of tokens the rule is a handful of small matrix products instead (the chunkwise form of delta rules with scalar gates: Yang,
// Kautz and Hatamizadeh, "Gated Delta Networks: Improving Mamba2 with Delta Rule"). With S the state in front of the chunk,
// D_ij the sum of the logarithms of the decays of tokens j + 1 .. i, e_i the product of the decays up to token i:
//   u_i = beta_i (v_i - e_i S^T k_i - sum_{j < i} exp(D_ij) (k_j . k_i) u_j)        (what token i writes)
//   o_i = e_i S^T q_i + sum_{j <= i} exp(D_ij) (k_j . q_i) u_j,   S <- e_last S + sum_j exp(D_last,j) k_j u_j^T,
// that is, with L_ij = beta_i exp(D_ij) k_j . k_i (j < i) and T = (I + L)^-1:  U = T diag(beta) (V - diag(e) K S),
// O = diag(e) Q S + A U. T and A do not depend on S: `delta_chunk_prepare` works them out for all chunks side by side, and
// `delta_chunks` walks a head's chunks with a tile of the state's columns in shared memory. Everything is 32-bit FMAs (no
// reduced-precision tensor-core mode): state, decays and gates stay what they are token by token, up to the order of sums.
// The logarithms D_ij are summed pair by pair from token j on, not taken as differences of sums from the chunk's start, so strong
// decays in front of a pair cost it no digits.
#include <type_traits>

#include "common.cuh"

namespace {

constexpr int C = 32;              // tokens per chunk
constexpr int kColumns = 16;       // columns of the state per block of `delta_chunks`
constexpr int kPrepareThreads = 256;
constexpr int kWalkThreads = 512;  // 16 warps: a block is alone on its SM for one request, so its own warps have to hide latencies
constexpr int kRowA = C + 4;       // row length of the 32 x 32 matrices in shared memory
constexpr int kRowS = kColumns + 4;

template <int kBytes>
__device__ __forceinline__ void stage_copy(float* smem, const float* gmem, bool valid) {
  const uint32_t s = static_cast<uint32_t>(__cvta_generic_to_shared(smem));
  const int bytes = valid ? kBytes : 0;
  asm volatile("cp.async.ca.shared.global [%0], [%1], %2, %3;" ::"r"(s), "l"(gmem), "n"(kBytes), "r"(bytes) : "memory");
}

// Rows `first .. first + n` of src [tokens][ld] from column `at` on, `width` numbers each, to dst [C][dst_ld], a warp per row; rows
// past n and columns from `width` to `padded` become zeros. W numbers a copy.
template <int W, int WARPS>
__device__ __forceinline__ void stage_rows(float* dst, int dst_ld, const float* src, int64_t first, int n, int64_t ld, int64_t at, int width, int padded) {
  const int lane = threadIdx.x & 31;
  for (int r = threadIdx.x >> 5; r < C; r += WARPS) {
    const float* from = src + (r < n ? (first + r) * ld + at : 0);
    for (int c = lane * W; c < padded; c += 32 * W) {
      const bool valid = r < n && c < width;
      stage_copy<4 * W>(dst + r * dst_ld + c, valid ? from + c : src, valid);
    }
  }
}

__host__ __device__ constexpr int padded_rows(int dk) { return (dk + 31) / 32 * 32; }

// One block per (chunk, q/k head, request); its warps take the heads that share the q/k head in turn.
// attn[t][head][j] = exp(D_ij) k_j . q_i (j <= i), solve[t][head][j] = T_ij beta_j, factors[t][head] = (e_i, exp(D_last,i)),
// for token t the i-th of its chunk.
template <int W>
__global__ void __launch_bounds__(kPrepareThreads)
delta_chunk_prepare_kernel(const float* q, const float* k, const float* beta, const float* log_decay, const int* __restrict__ seq_q_start,
                           const int* __restrict__ seq_q_len, int heads, int kv_heads, int dk, float* attn, float* solve, float* factors) {
  extern __shared__ __align__(16) float chunk_smem[];
  let_successor_start();
  const int seq = blockIdx.z, kvh = blockIdx.y, chunk = blockIdx.x;
  const int len = seq_q_len[seq], n = min(C, len - chunk * C);
  if (n <= 0) return;
  const int64_t first = static_cast<int64_t>(seq_q_start[seq]) + chunk * C;
  const int padded = padded_rows(dk), ld = padded + 4;
  float* ks = chunk_smem;           // [C][ld]
  float* qs = ks + C * ld;          // [C][ld]
  float* kk = qs + C * ld;          // [C][C + 1]: k_i . k_j
  float* qk = kk + C * (C + 1);     // [C][C + 1]: q_i . k_j
  float* ls = qk + C * (C + 1);     // [warps][C][C]: L of the head a warp works on
  wait_for_predecessor();
  constexpr int kWarps = kPrepareThreads / 32;
  stage_rows<W, kWarps>(ks, ld, k, first, n, static_cast<int64_t>(kv_heads) * dk, static_cast<int64_t>(kvh) * dk, dk, padded);
  stage_rows<W, kWarps>(qs, ld, q, first, n, static_cast<int64_t>(kv_heads) * dk, static_cast<int64_t>(kvh) * dk, dk, padded);
  asm volatile("cp.async.commit_group;\ncp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  {
    // A warp has rows 4 warp .. + 3 of both products; a thread every fourth group of four channels and columns j0, j0 + 8, ..,
    // as far as the triangle reaches.
    const int j0 = tid & 7, part = (tid >> 3) & 3, i0 = warp * 4;
    const int reach = (i0 + 3) / 8;  // last x whose columns j0 + 8 x the triangle needs
    float acc[8][4];                 // k_i . k_j of four rows, then q_i . k_j
#pragma unroll
    for (int r = 0; r < 8; ++r) acc[r][0] = acc[r][1] = acc[r][2] = acc[r][3] = 0.f;
    for (int c = part * 4; c < padded; c += 16) {
      float4 rows[8];
#pragma unroll
      for (int r = 0; r < 4; ++r) {
        rows[r] = *reinterpret_cast<const float4*>(ks + (i0 + r) * ld + c);
        rows[r + 4] = *reinterpret_cast<const float4*>(qs + (i0 + r) * ld + c);
      }
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        if (x > reach) break;
        const float4 kj = *reinterpret_cast<const float4*>(ks + (j0 + 8 * x) * ld + c);
#pragma unroll
        for (int r = 0; r < 8; ++r)
          acc[r][x] = fmaf(rows[r].x, kj.x, fmaf(rows[r].y, kj.y, fmaf(rows[r].z, kj.z, fmaf(rows[r].w, kj.w, acc[r][x]))));
      }
    }
    // The four parts meet: a lane ends with two rows of one product.
    const bool b0 = part & 1, b1 = part & 2;
    float* product = (b0 ? qk : kk) + (i0 + (b1 ? 2 : 0)) * (C + 1);
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      float half[4];
#pragma unroll
      for (int r = 0; r < 4; ++r) half[r] = (b0 ? acc[r + 4][x] : acc[r][x]) + __shfl_xor_sync(0xffffffffu, b0 ? acc[r][x] : acc[r + 4][x], 8);
#pragma unroll
      for (int r = 0; r < 2; ++r)
        product[r * (C + 1) + j0 + 8 * x] = (b1 ? half[r + 2] : half[r]) + __shfl_xor_sync(0xffffffffu, b1 ? half[r] : half[r + 2], 16);
    }
  }
  __syncthreads();
  const int group = heads / kv_heads;
  float* mine = ls + warp * C * C;
  for (int g = 0; g < group; ++g) {
    const int head = kvh * group + g;
    const int64_t at = (first + lane) * heads + head;
    const float own = lane < n ? log_decay[at] : 0.f;
    const float own_beta = lane < n ? beta[at] : 0.f;
    const bool solves = (g & 7) == warp;
    // Column j = lane: D_ij grows with i from zero at i = j.
    float d = 0.f, prefix = 0.f, e = 0.f;
    for (int i = 0; i < C; ++i) {
      const float gi = __shfl_sync(0xffffffffu, own, i), bi = __shfl_sync(0xffffffffu, own_beta, i);
      d = i > lane ? d + gi : 0.f;
      prefix += gi;
      if (i == lane) e = prefix;
      if ((i & 7) == warp && i < n)
        attn[((first + i) * heads + head) * C + lane] = lane <= i ? expf(d) * qk[i * (C + 1) + lane] : 0.f;
      if (solves) mine[i * C + lane] = lane < i ? bi * expf(d) * kk[i * (C + 1) + lane] : 0.f;
    }
    if (!solves) continue;
    // d is now D_last,j: tokens past n added nothing.
    if (lane < n) *reinterpret_cast<float2*>(factors + at * 2) = make_float2(expf(e), expf(d));
    __syncwarp();
    // T = (I + L)^-1 by forward substitution, column j on lane j: T_i = delta_ij - sum_{m < i} L_im T_m.
    float t[C];
#pragma unroll
    for (int i = 0; i < C; ++i) {
      float sum0 = i == lane ? 1.f : 0.f, sum1 = 0.f;
#pragma unroll
      for (int m = 0; m < i; m += 4) {
        const float4 l = *reinterpret_cast<const float4*>(mine + i * C + m);
        sum0 = fmaf(-l.x, t[m], sum0);
        if (m + 1 < i) sum1 = fmaf(-l.y, t[m + 1], sum1);
        if (m + 2 < i) sum0 = fmaf(-l.z, t[m + 2], sum0);
        if (m + 3 < i) sum1 = fmaf(-l.w, t[m + 3], sum1);
      }
      t[i] = sum0 + sum1;
      if (i < n) solve[((first + i) * heads + head) * C + lane] = t[i] * own_beta;
    }
    __syncwarp();
  }
}

// Partial sums of four rows by four columns on eight lanes (lane bits 2, 3, 4 count them) -> the whole sums of two neighbouring
// columns of one row each: row 2 b2 + b3, columns 2 b4 and 2 b4 + 1.
__device__ __forceinline__ float2 gather_pair(const float (&acc)[4][4], int lane) {
  const bool b2 = lane & 4, b3 = lane & 8, b4 = lane & 16;
  float two[2][4], row[4];
#pragma unroll
  for (int r = 0; r < 2; ++r)
#pragma unroll
    for (int c = 0; c < 4; ++c) two[r][c] = (b2 ? acc[r + 2][c] : acc[r][c]) + __shfl_xor_sync(0xffffffffu, b2 ? acc[r][c] : acc[r + 2][c], 4);
#pragma unroll
  for (int c = 0; c < 4; ++c) row[c] = (b3 ? two[1][c] : two[0][c]) + __shfl_xor_sync(0xffffffffu, b3 ? two[0][c] : two[1][c], 8);
  return make_float2((b4 ? row[2] : row[0]) + __shfl_xor_sync(0xffffffffu, b4 ? row[0] : row[2], 16),
                     (b4 ? row[3] : row[1]) + __shfl_xor_sync(0xffffffffu, b4 ? row[1] : row[3], 16));
}

__device__ __forceinline__ void fma_row(float (&acc)[4], float a, const float4& s) {
  acc[0] = fmaf(a, s.x, acc[0]), acc[1] = fmaf(a, s.y, acc[1]), acc[2] = fmaf(a, s.z, acc[2]), acc[3] = fmaf(a, s.w, acc[3]);
}

__host__ __device__ constexpr int stage_floats(int padded) { return 2 * C * (padded + 4) + C * kRowS + 2 * C * kRowA + 2 * C; }
constexpr size_t chunks_smem(int padded) { return sizeof(float) * (2 * stage_floats(padded) + padded * kRowS + 4 * C * kRowS); }

// One block per (16 columns of the state, head, request); the next chunk's operands arrive by cp.async while one is worked on.
template <int W>
__global__ void __launch_bounds__(kWalkThreads, 2)
delta_chunks_kernel(const float* q, const float* k, const float* v, const float* attn, const float* solve, const float* factors,
                    const int* __restrict__ seq_q_start, const int* __restrict__ seq_q_len, const int* __restrict__ seq_slot, int heads, int kv_heads,
                    int dk, int dv, float* state, float* out) {
  extern __shared__ __align__(16) float chunk_smem[];
  let_successor_start();
  const int col0 = blockIdx.x * kColumns, head = blockIdx.y, seq = blockIdx.z;
  const int kvh = head / (heads / kv_heads);
  const int64_t start = seq_q_start[seq];
  const int len = seq_q_len[seq];
  const int padded = padded_rows(dk), ld = padded + 4;
  const int columns = min(kColumns, dv - col0);
  const int tid = threadIdx.x, lane = tid & 31;
  const int per_stage = stage_floats(padded);
  float* S = chunk_smem + 2 * per_stage;  // [padded][kRowS]
  float* X = S + padded * kRowS;          // [C][kRowS]: V - diag(e) K S
  float* R = X + C * kRowS;               // diag(e) Q S
  float* U = R + C * kRowS;
  float* Ud = U + C * kRowS;              // [C][kColumns]: exp(D_last,j) u_j
  float* s_base = state + (static_cast<int64_t>(seq_slot[seq]) * heads + head) * dk * dv + col0;
  wait_for_predecessor();
  auto fetch = [&](int buffer, int chunk) {
    float* ks = chunk_smem + buffer * per_stage;
    float* qs = ks + C * ld;
    float* vs = qs + C * ld;
    float* as = vs + C * kRowS;
    float* ws = as + C * kRowA;
    float* fs = ws + C * kRowA;
    const int n = min(C, len - chunk * C);
    const int64_t first = start + chunk * C;
    constexpr int kWarps = kWalkThreads / 32;
    stage_rows<W, kWarps>(ks, ld, k, first, n, static_cast<int64_t>(kv_heads) * dk, static_cast<int64_t>(kvh) * dk, dk, padded);
    stage_rows<W, kWarps>(qs, ld, q, first, n, static_cast<int64_t>(kv_heads) * dk, static_cast<int64_t>(kvh) * dk, dk, padded);
    {  // both 32 x 32 matrices, 16 bytes a thread
      const int r = (tid >> 3) & 31, c = (tid & 7) * 4;
      const int64_t at = ((first + r) * heads + head) * C + c;
      stage_copy<16>((tid < 256 ? as : ws) + r * kRowA + c, (tid < 256 ? attn : solve) + (r < n ? at : 0), r < n);
    }
    if (tid < C * kColumns / W) {
      const int r = tid / (kColumns / W), c = tid % (kColumns / W) * W;
      const bool valid = r < n && c < columns;
      stage_copy<4 * W>(vs + r * kRowS + c, v + (valid ? ((first + r) * heads + head) * dv + col0 + c : 0), valid);
    }
    if (tid >= kWalkThreads - 2 * C) {
      const int x = tid - (kWalkThreads - 2 * C), r = x >> 1;
      stage_copy<4>(fs + x, factors + (r < n ? ((first + r) * heads + head) * 2 + (x & 1) : 0), r < n);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if (len > 0) fetch(0, 0);
  for (int idx = tid; idx < padded * kColumns; idx += kWalkThreads) {
    const int r = idx / kColumns, c = idx % kColumns;
    S[r * kRowS + c] = r < dk && c < columns ? s_base[static_cast<int64_t>(r) * dv + c] : 0.f;
  }
  const int chunks = (len + C - 1) / C;
  for (int chunk = 0; chunk < chunks; ++chunk) {
    const int n = min(C, len - chunk * C);
    if (chunk + 1 < chunks) {
      fetch((chunk + 1) & 1, chunk + 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const float* ks = chunk_smem + (chunk & 1) * per_stage;
    const float* qs = ks + C * ld;
    const float* vs = qs + C * ld;
    const float* as = vs + C * kRowS;
    const float* ws = as + C * kRowA;
    const float* fs = ws + C * kRowA;
    {
      // K S and Q S: a thread has four rows of [K; Q] and four columns, and every eighth group of four rows of S. The lanes that
      // load together (eight for 16-byte accesses) read two neighbouring groups' rows over all four groups of columns.
      const int ct = tid & 3, part = (tid >> 2) & 7, rt = tid >> 5;
      const float* rows = (rt < 8 ? ks : qs) + (rt & 7) * 4 * ld + part * 4;
      const float* cols = S + part * 4 * kRowS + ct * 4;
      float acc[4][4];
#pragma unroll
      for (int r = 0; r < 4; ++r) acc[r][0] = acc[r][1] = acc[r][2] = acc[r][3] = 0.f;
#pragma unroll 2
      for (int c = 0; c < padded; c += 32) {
        float4 a[4], s[4];
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          a[x] = *reinterpret_cast<const float4*>(rows + x * ld + c);
          s[x] = *reinterpret_cast<const float4*>(cols + (c + x) * kRowS);
        }
#pragma unroll
        for (int r = 0; r < 4; ++r) {
          fma_row(acc[r], a[r].x, s[0]);
          fma_row(acc[r], a[r].y, s[1]);
          fma_row(acc[r], a[r].z, s[2]);
          fma_row(acc[r], a[r].w, s[3]);
        }
      }
      const float2 sum = gather_pair(acc, lane);
      const int i = (rt & 7) * 4 + ((lane >> 2) & 1) * 2 + ((lane >> 3) & 1), at = i * kRowS + ct * 4 + ((lane >> 4) & 1) * 2;
      const float e = fs[2 * i];
      if (rt < 8) {
        const float2 value = *reinterpret_cast<const float2*>(vs + at);
        *reinterpret_cast<float2*>(X + at) = make_float2(fmaf(-e, sum.x, value.x), fmaf(-e, sum.y, value.y));
      } else {
        *reinterpret_cast<float2*>(R + at) = make_float2(e * sum.x, e * sum.y);
      }
    }
    __syncthreads();
    // Products with the lower triangular 32 x 32 matrices: sum_{m <= i} matrix[i][m] operand[m][c2, c2 + 1], over every `step`-th
    // group of four m from `from` on (zeros follow m = i).
    auto triangle = [&](const float* matrix, const float* operand, int i, int c2, int from, int step) {
      float2 sum = make_float2(0.f, 0.f);
#pragma unroll 2
      for (int m = from; m <= (i & ~3); m += step) {
        const float4 w = *reinterpret_cast<const float4*>(matrix + i * kRowA + m);
        const float factor[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const float2 u = *reinterpret_cast<const float2*>(operand + (m + x) * kRowS + c2);
          sum.x = fmaf(factor[x], u.x, sum.x), sum.y = fmaf(factor[x], u.y, sum.y);
        }
      }
      return sum;
    };
    {
      const int i = tid >> 4, c2 = (tid & 7) * 2, half = (tid >> 3) & 1;
      float2 u = triangle(ws, X, i, c2, half * 4, 8);
      u.x += __shfl_xor_sync(0xffffffffu, u.x, 8);
      u.y += __shfl_xor_sync(0xffffffffu, u.y, 8);
      const float d = fs[2 * i + 1];
      if (half == 0) *reinterpret_cast<float2*>(U + i * kRowS + c2) = u;
      else *reinterpret_cast<float2*>(Ud + i * kColumns + c2) = make_float2(d * u.x, d * u.y);
    }
    __syncthreads();
    if (tid >= 256) {  // half of the warps: the outputs; the other half moves the state on
      const int i = (tid - 256) >> 3, c2 = (tid & 7) * 2;
      if (i < n) {
        const float2 o = triangle(as, U, i, c2, 0, 4);
        float* to = out + ((start + chunk * C + i) * heads + head) * dv + col0 + c2;
        if (c2 < columns) to[0] = R[i * kRowS + c2] + o.x;
        if (c2 + 1 < columns) to[1] = R[i * kRowS + c2 + 1] + o.y;
      }
    } else {
      // S <- e_last S + K^T (exp(D_last) U): four rows and four columns a thread, half of the tokens each.
      const float last = fs[2 * (n - 1)];
      const int part = tid & 1, ct = (tid >> 1) & 3;
      for (int tile = tid >> 3; tile * 4 < padded; tile += 32) {
        float acc[4][4];
#pragma unroll
        for (int r = 0; r < 4; ++r) acc[r][0] = acc[r][1] = acc[r][2] = acc[r][3] = 0.f;
#pragma unroll 4
        for (int j = part; j < C; j += 2) {
          const float4 kj = *reinterpret_cast<const float4*>(ks + j * ld + tile * 4);
          const float4 uj = *reinterpret_cast<const float4*>(Ud + j * kColumns + ct * 4);
          fma_row(acc[0], kj.x, uj);
          fma_row(acc[1], kj.y, uj);
          fma_row(acc[2], kj.z, uj);
          fma_row(acc[3], kj.w, uj);
        }
#pragma unroll
        for (int r = 0; r < 2; ++r) {  // the two lanes of a tile keep two rows each
          float whole[4];
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            const float give = part ? acc[r][c] : acc[r + 2][c], keep = part ? acc[r + 2][c] : acc[r][c];
            whole[c] = keep + __shfl_xor_sync(0xffffffffu, give, 1);
          }
          float4* at = reinterpret_cast<float4*>(S + (tile * 4 + part * 2 + r) * kRowS + ct * 4);
          const float4 old = *at;
          *at = make_float4(fmaf(last, old.x, whole[0]), fmaf(last, old.y, whole[1]), fmaf(last, old.z, whole[2]), fmaf(last, old.w, whole[3]));
        }
      }
    }
    __syncthreads();  // the state is the next chunk's, this chunk's stage is free
  }
  for (int idx = tid; idx < dk * kColumns; idx += kWalkThreads) {
    const int r = idx / kColumns, c = idx % kColumns;
    if (c < columns && len > 0) s_base[static_cast<int64_t>(r) * dv + c] = S[r * kRowS + c];
  }
}

size_t prepare_smem(int padded) { return sizeof(float) * (2 * C * (padded + 4) + 2 * C * (C + 1) + (kPrepareThreads / 32) * C * C); }

}  // namespace

constexpr int kChunkMaxRows = 256;

// Key sizes whose chunks fit shared memory; the caller walks token by token otherwise.
B200_API int b200_delta_chunks_supported(int heads, int kv_heads, int dk, int dv) {
  return heads > 0 && heads <= 65535 && kv_heads > 0 && heads % kv_heads == 0 && dk > 0 && dk <= kChunkMaxRows && dv > 0;
}

// Scratch: `attn` and `solve` [tokens][heads][32], `factors` [tokens][heads][2]. The other operands are those of
// b200_delta_head_recurrence.
B200_API int b200_delta_chunks(const float* q, const float* k, const float* v, const float* beta, const float* log_decay, const int* seq_q_start,
                               const int* seq_q_len, const int* seq_slot, int seqs, int max_q_len, int heads, int kv_heads, int dk, int dv, float* attn,
                               float* solve, float* factors, float* state, float* out, cudaStream_t stream) {
  if (seqs == 0) return 0;
  B200_REQUIRE(seqs > 0 && seqs <= 65535 && max_q_len > 0 && b200_delta_chunks_supported(heads, kv_heads, dk, dv), "delta_chunks: shape not taken");
  const auto aligned = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
  B200_REQUIRE(aligned(attn) && aligned(solve) && aligned(factors), "delta_chunks: scratch must be aligned to 16 bytes");
  const bool wide = dk % 4 == 0 && dv % 4 == 0 && aligned(q) && aligned(k) && aligned(v);
  const int padded = padded_rows(dk);
  const size_t prepare_bytes = prepare_smem(padded), walk_bytes = chunks_smem(padded);
  auto raise = [](auto kernel, size_t bytes) {
    return cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(bytes)) == cudaSuccess;
  };
  static bool raised = false;
  if (!raised) {
    const size_t a = prepare_smem(kChunkMaxRows), b = chunks_smem(kChunkMaxRows);
    if (!raise(delta_chunk_prepare_kernel<1>, a) || !raise(delta_chunk_prepare_kernel<4>, a) || !raise(delta_chunks_kernel<1>, b) ||
        !raise(delta_chunks_kernel<4>, b))
      return b200_fail("delta_chunks: cannot size shared memory");
    raised = true;
  }
  const dim3 prepare_grid((max_q_len + C - 1) / C, kv_heads, seqs), walk_grid((dv + kColumns - 1) / kColumns, heads, seqs);
  launch_kernel(wide ? delta_chunk_prepare_kernel<4> : delta_chunk_prepare_kernel<1>, prepare_grid, dim3(kPrepareThreads), prepare_bytes, stream, q, k, beta,
                log_decay, seq_q_start, seq_q_len, heads, kv_heads, dk, attn, solve, factors);
  if (int status = b200_check_launch("delta_chunk_prepare")) return status;
  // The ordinary way, not early: the few long-lived blocks should spread over all SMs, not over those the kernel in front leaves first.
  launch_kernel_as(true, wide ? delta_chunks_kernel<4> : delta_chunks_kernel<1>, walk_grid, dim3(kWalkThreads), walk_bytes, stream, q, k, v, attn, solve,
                   factors, seq_q_start, seq_q_len, seq_slot, heads, kv_heads, dk, dv, state, out);
  return b200_check_launch("delta_chunks");
}
