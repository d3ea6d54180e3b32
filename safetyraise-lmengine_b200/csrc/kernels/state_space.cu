// A state space with one decay a head (the second Mamba's recurrence), on a matrix of state S [N, P] per head and request:
//
//   S <- exp(-exp(A_h) dt) S + dt B x^T;   y = S^T C + D_h x            dt = softplus(dt_in + bias), no clamp
//
// x (P a head), B and C (N each, shared by the heads of a group) behind one short causal convolution with a bias and silu.
// Then y * silu(z), normed over equal parts of the heads' concatenation, times a weight.  Everything behind the projection
// is float32.
//
// proj float32 [T, ldp]: z (H P) | x (H P) | B (G N) | C (G N) | dt (H).  The convolution's channels are x | B | C.
// A request's state row: S [H][P][N] (a column of S contiguous) | the last taps - 1 inputs of the convolution's channels
// ([taps - 1][channels], renewed by conv_carry behind the kernels that read them).
//
//   state_space_walk     token by token: convolution, step size, recurrence in one launch; any sizes (decoding)
//   state_space_groups   for every group of 8 tokens and head, what all columns of S share: with P_i = the product of the
//                        decays up to token i of the group and R_j = the product of those behind token j,
//                          M_ij = (C_i . B_j) decay_(j+1) .. decay_i dt_j (j <= i),  P_i,  R_j dt_j
//   state_space_read     walks the groups with S in registers:
//                          y_i = P_i (C_i . S) + sum_j M_ij x_j + D x_i,   S <- P_8 S + sum_j B_j (R_j dt_j x_j)
//   state_space_output   gate, norm of each part, weight, rounding
#include "state_walk.cuh"

namespace srlm {

struct SpaceSizes {
  int H, G, N, P;
};

template <int RPL>
__global__ void __launch_bounds__(RPL <= 32 ? 512 : 256)
state_space_walk_kernel(ConvInput in, const float* __restrict__ conv_w, const float* __restrict__ conv_b,
                        const float* __restrict__ dt_in, const float* __restrict__ dt_bias, const float* __restrict__ a_log,
                        const float* __restrict__ D, float* __restrict__ state, const int* __restrict__ cu_q,
                        const int* __restrict__ slots, float* __restrict__ y_out, SpaceSizes z, int cols, int vec) {
  constexpr int NP = RPL * kStateLanes;
  extern __shared__ __align__(16) float walk_smem[];
  float* b_s = walk_smem;                    // [NP] each, zeros behind N
  float* c_s = b_s + NP;
  float* x_s = c_s + NP;                     // [cols]
  const int e = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * cols, tid = threadIdx.x;
  const int cg = tid / kStateLanes, l = tid % kStateLanes, col = c0 + cg;
  const bool live = col < z.P;
  const int grp = h / (z.H / z.G), width = min(cols, z.P - c0);
  const int slot = slots[e];
  float* S_col = state + (size_t)slot * in.state_stride + ((size_t)h * z.P + (live ? col : 0)) * z.N;
  float S[RPL];
  pdl_wait();
  pdl_trigger();
  load_column<RPL>(S, S_col, l, z.N, live, vec);
  const float rate = expf(a_log[h]), d_h = D[h], bias = dt_bias[h];
  const int t0 = cu_q[e], n = cu_q[e + 1] - t0;
  for (int i = tid; i < 2 * NP; i += blockDim.x) walk_smem[i] = 0.f;
  for (int i = 0; i < n; ++i) {
    const int t = t0 + i;
    __syncthreads();                         // the token before is no longer read
    for (int x = tid; x < 2 * z.N + width; x += blockDim.x) {
      const int part = x / z.N;
      const int c = part == 0 ? z.H * z.P + grp * z.N + x : part == 1 ? z.H * z.P + (z.G + grp) * z.N + (x - z.N)
                                                                     : h * z.P + c0 + (x - 2 * z.N);
      const float y = silu_of(conv_at(in, conv_w, t, i, slot, c) + conv_b[c]);
      (part == 0 ? b_s + x : part == 1 ? c_s + (x - z.N) : x_s + (x - 2 * z.N))[0] = y;
    }
    const float dt = softplus_f(dt_in[(size_t)t * in.ld + h] + bias);
    const float keep = expf(-rate * dt);
    __syncthreads();
    const float xv = live ? x_s[cg] : 0.f, w = dt * xv;
    float2 b2 = make_float2(0.f, 0.f);
#pragma unroll
    for (int j = 0; j < RPL / 4; ++j) {
      const float4 bv = *reinterpret_cast<const float4*>(b_s + 32 * j + 4 * l);
      const float4 cv = *reinterpret_cast<const float4*>(c_s + 32 * j + 4 * l);
      S[4 * j] = fmaf(bv.x, w, keep * S[4 * j]);
      S[4 * j + 1] = fmaf(bv.y, w, keep * S[4 * j + 1]);
      S[4 * j + 2] = fmaf(bv.z, w, keep * S[4 * j + 2]);
      S[4 * j + 3] = fmaf(bv.w, w, keep * S[4 * j + 3]);
      b2 = fma2(make_float2(cv.x, cv.y), make_float2(S[4 * j], S[4 * j + 1]), b2);
      b2 = fma2(make_float2(cv.z, cv.w), make_float2(S[4 * j + 2], S[4 * j + 3]), b2);
    }
    float y = b2.x + b2.y;
#pragma unroll
    for (int o = 1; o < kStateLanes; o <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
    if (live && l == 0) y_out[((size_t)t * z.H + h) * z.P + col] = fmaf(d_h, xv, y);
  }
  store_column<RPL>(S, S_col, l, z.N, live, vec);
}

// ---- groups of 8 tokens ------------------------------------------------------------------------------------------------
// A group's record for one head, floats: M [8][8] | P [8] | R dt [8].
constexpr int kSpaceRecord = kStateGroup * kStateGroup + 2 * kStateGroup;

// A warp per (group, head).  conv: the convolved and activated x | B | C channels, float32 [T, C].
__global__ void __launch_bounds__(128)
state_space_groups_kernel(const float* __restrict__ conv, int C, const float* __restrict__ dt_in, long long ldp,
                          const float* __restrict__ dt_bias, const float* __restrict__ a_log, const int* __restrict__ cu_q,
                          int n_entries, float* __restrict__ records, SpaceSizes z) {
  pdl_wait();
  pdl_trigger();
  constexpr int M = kStateGroup;
  __shared__ float sums[4][64];
  __shared__ float steps[4][2 * M];          // dt_i, decay_i
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int h = blockIdx.y * 4 + warp;
  const GroupHome home = group_home(cu_q, n_entries, blockIdx.x);
  if (home.entry < 0 || h >= z.H) return;
  const int grp = h / (z.H / z.G);
  if (lane < M) {
    const bool there = lane < home.n;
    const float dt = there ? softplus_f(dt_in[(size_t)(home.t0 + lane) * ldp + h] + dt_bias[h]) : 0.f;
    steps[warp][lane] = dt;
    steps[warp][M + lane] = there ? expf(-expf(a_log[h]) * dt) : 1.f;
  }
  float acc[64];                             // C_i . B_j at 8 i + j; only j <= i is filled
#pragma unroll
  for (int s = 0; s < 64; ++s) acc[s] = 0.f;
  const float* first = conv + (size_t)home.t0 * C + (size_t)z.H * z.P + (size_t)grp * z.N;
  for (int r = lane; r < z.N; r += 32) {
    float b[M], c[M];
#pragma unroll
    for (int i = 0; i < M; ++i) {
      const bool there = i < home.n;
      b[i] = there ? first[(size_t)i * C + r] : 0.f;
      c[i] = there ? first[(size_t)i * C + (size_t)z.G * z.N + r] : 0.f;
    }
#pragma unroll
    for (int i = 0; i < M; ++i)
#pragma unroll
      for (int j = 0; j <= i; ++j) acc[8 * i + j] = fmaf(c[i], b[j], acc[8 * i + j]);
  }
  scatter_sums<64, 32>(acc, lane);
  const int at = 2 * lane;
  sums[warp][at] = acc[0];
  sums[warp][at + 1] = acc[1];
  __syncwarp();
  float* rec = records + ((size_t)blockIdx.x * z.H + h) * kSpaceRecord;
#pragma unroll
  for (int x = lane; x < M * M; x += 32) {
    const int i = x / M, j = x % M;
    float f = steps[warp][j];
    for (int s = j + 1; s <= i; ++s) f *= steps[warp][M + s];
    rec[x] = j <= i ? sums[warp][x] * f : 0.f;
  }
  if (lane < M) {
    float pre = 1.f, suf = steps[warp][lane];
    for (int s = 0; s <= lane; ++s) pre *= steps[warp][M + s];
    for (int s = lane + 1; s < M; ++s) suf *= steps[warp][M + s];
    rec[M * M + lane] = pre;
    rec[M * M + M + lane] = suf;
  }
}

constexpr int kSpaceCols = 16, kSpaceStages = 3, kSpaceThreads = 128;  // 128 = 8 tokens x 16 columns: a value a thread

// Block: 16 columns of one head's S for one entry, four a warp.
template <int NP, int L>
__global__ void __launch_bounds__(kSpaceThreads, 4)     // four blocks an SM: up to 128 registers, loads in flight
state_space_read_kernel(const float* __restrict__ records, const float* __restrict__ conv, int C, const float* __restrict__ D,
                        float* __restrict__ state, long long state_stride, const int* __restrict__ cu_q,
                        const int* __restrict__ slots, float* __restrict__ y_out, SpaceSizes z, int vec, int vec_rows) {
  pdl_wait();
  pdl_trigger();
  typedef StateTile<NP, L> Tile;
  constexpr int M = kStateGroup, STAGE = 2 * M * NP + kSpaceRecord + M * kSpaceCols, NC = Tile::kColumns;
  extern __shared__ __align__(16) float read_smem[];        // [kSpaceStages]: C rows [8][NP] | B rows [8][NP] | the record | x [8][16]
  __shared__ __align__(16) float w_s[kSpaceThreads / 32][32 * NC];
  const int e = blockIdx.z, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int grp = h / (z.H / z.G);
  const int hl = lane % L, set = lane / L, l = lane & 7;
  const int col_set = blockIdx.x * kSpaceCols + 4 * warp + set * NC;       // the first column that the lane holds rows of
  const int col = blockIdx.x * kSpaceCols + 4 * warp + (lane >> 3);        // the column whose token l the lane finishes
  const bool live = col < z.P;
  const int t0 = cu_q[e], n = cu_q[e + 1] - t0, groups = (n + M - 1) / M;
  const float* rec0 = records + ((size_t)first_group(cu_q, e) * z.H + h) * kSpaceRecord;
  const float* rows0 = conv + (size_t)t0 * C + (size_t)z.H * z.P + (size_t)grp * z.N;
  for (int i = tid; i < kSpaceStages * STAGE; i += kSpaceThreads) read_smem[i] = 0.f;
  __syncthreads();                           // rows behind N and tokens behind the portion stay zero (or finite)
  constexpr int kCopies = 2 * M * NP / 4 / kSpaceThreads;   // a thread's 16-byte pieces of a group's rows
  int copy_to[kCopies], copy_tok[kCopies];
  unsigned copy_from[kCopies];
#pragma unroll
  for (int i = 0; i < kCopies; ++i) {
    const int x = tid + i * kSpaceThreads, pieces = z.N / 4, row = pieces ? x / pieces : 2 * M, at = (x - row * pieces) * 4;
    copy_tok[i] = row < 2 * M ? row % M : M;                // M: no piece
    copy_to[i] = row * NP + at;
    copy_from[i] = (unsigned)(row % M) * (unsigned)C + (row < M ? (unsigned)(z.G * z.N) : 0u) + (unsigned)at;
  }
  const int x_col = blockIdx.x * kSpaceCols + tid % kSpaceCols;
  const float* x_in = conv + (size_t)h * z.P + x_col;
  auto fetch = [&](int g) {
    if (g < groups) {
      float* dst = read_smem + (g % kSpaceStages) * STAGE;
      const int m = min(M, n - g * M);
      const float* src = rows0 + (size_t)g * M * C;
      if (vec_rows) {
#pragma unroll
        for (int i = 0; i < kCopies; ++i)
          if (copy_tok[i] < m) state_copy_16(dst + copy_to[i], src + copy_from[i]);
      } else {
        for (int i = tid; i < 2 * M * z.N; i += kSpaceThreads) {
          const int row = i / z.N, x = i - row * z.N, tok = row % M;
          if (tok < m)
            state_copy_4(dst + row * NP + x, src + (size_t)tok * C + (row < M ? (size_t)z.G * z.N : 0) + x);
        }
      }
      if (tid < kSpaceRecord / 4) state_copy_16(dst + 2 * M * NP + 4 * tid, rec0 + (size_t)g * z.H * kSpaceRecord + 4 * tid);
      const int tok = tid / kSpaceCols;                     // a thread's value of the group
      float* x_at = dst + 2 * M * NP + kSpaceRecord + tid;
      if (tok < m && x_col < z.P) state_copy_4(x_at, x_in + (size_t)(t0 + g * M + tok) * C);
      else *x_at = 0.f;
    }
    state_copy_commit();
  };
  fetch(0);
  fetch(1);
  const float d_h = D[h];
  float* S_head = state + (size_t)slots[e] * state_stride + (size_t)h * z.P * z.N;
  Tile S;
  S.load(S_head, col_set, z.P, hl, z.N, vec);
  int row_of[M];                             // where the lane's piece of the vector of token slot i lies
#pragma unroll
  for (int i = 0; i < M; ++i) row_of[i] = (i ^ l) * NP + 4 * hl;
  for (int g = 0; g < groups; ++g) {
    state_copy_wait<1>();
    __syncthreads();                         // group g is here for all; group g - 1 is read by all
    fetch(g + 2);
    const float* st = read_smem + (g % kSpaceStages) * STAGE;
    const float* rec = st + 2 * M * NP;
    const float x = rec[kSpaceRecord + l * kSpaceCols + 4 * warp + (lane >> 3)];
    float p[8 * NC];                         // slots of column c and token i: C_i . S at 8 c + i
#pragma unroll
    for (int i = 0; i < M; ++i) {
      float b[NC];
      S.dot(st + row_of[i], b);
#pragma unroll
      for (int c = 0; c < NC; ++c) p[8 * c + i] = b[c];
    }
    Tile::share(w_s[warp], set, hl, rec[M * M + M + l] * x);
    permuted_sums<8 * NC, L>(p);
    float y = p[0] * rec[M * M + l] + d_h * x;
    const float4 m0 = *reinterpret_cast<const float4*>(rec + l * M), m1 = *reinterpret_cast<const float4*>(rec + l * M + 4);
    const float mr[M] = {m0.x, m0.y, m0.z, m0.w, m1.x, m1.y, m1.z, m1.w};
    __syncwarp();
    const float keep = rec[M * M + M - 1];
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
      for (int j = 0; j < 2 * Tile::kPieces; ++j) { S.s[c][j].x *= keep; S.s[c][j].y *= keep; }
#pragma unroll
    for (int j = 0; j < M; ++j) {
      alignas(16) float wj[NC];
      Tile::shared(w_s[warp], set, hl, j, wj);
      S.add(st + (M + j) * NP + 4 * hl, wj);
      y = fmaf(mr[j], __shfl_sync(0xffffffffu, x, j, M), y);
    }
    if (live && g * M + l < n) y_out[((size_t)(t0 + g * M + l) * z.H + h) * z.P + col] = y;
  }
  state_copy_wait<0>();
  S.store(S_head, col_set, z.P, hl, z.N, vec);
}

// A block per (part, token): out = w * u / sqrt(mean(u^2) + eps) over the part, u = y * silu(z).
template <typename TO>
__global__ void state_space_output_kernel(const float* __restrict__ y, const float* __restrict__ proj, long long ldp,
                                          const float* __restrict__ w, float eps, TO* __restrict__ out, int inner, int part) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ float out_smem[];        // [part]
  __shared__ float scratch[32];
  const size_t t = blockIdx.y;
  const int c0 = blockIdx.x * part;
  float ss = 0.f;
  for (int i = threadIdx.x; i < part; i += blockDim.x) {
    const float u = y[t * inner + c0 + i] * silu_of(proj[t * ldp + c0 + i]);
    out_smem[i] = u;
    ss += u * u;
  }
  const float inv = 1.f / sqrtf(block_sum(ss, scratch) / (float)part + eps);
  for (int i = threadIdx.x; i < part; i += blockDim.x)
    out[t * inner + c0 + i] = from_float<TO>(out_smem[i] * inv * w[c0 + i]);
}

}  // namespace srlm

using namespace srlm;

static int space_ok(const char* what, int H, int G, int N, int P, long long ldp, long long state_stride, int n_entries) {
  if (H <= 0 || G <= 0 || H % G || N <= 0 || N > 512 || P <= 0 || H > 65535 || n_entries > 65535 ||
      ldp < 2LL * H * P + 2LL * G * N + H || state_stride < (long long)H * N * P || (long long)H * N * P > 0x7fffffffLL)
    return refuse(ST_BAD_SIZE, "%s: heads=%d groups=%d state=%d (at most 512) vdim=%d ld=%lld row=%lld entries=%d", what, H, G, N, P,
                  ldp, state_stride, n_entries);
  return ST_OK;
}
static int rows_per_lane(int rows) { return rows <= 32 ? 4 : rows <= 64 ? 8 : rows <= 128 ? 16 : rows <= 256 ? 32 : 64; }

// proj as above; conv_w float32 [channels, taps], conv_b [channels]; dt_bias, a_log, D float32 [H]; y_out float32 [T, H P].
extern "C" int srlm_state_space_walk(const float* proj, long long ldp, const float* conv_w, const float* conv_b,
                                     const float* dt_bias, const float* a_log, const float* D, float* state,
                                     long long state_stride, const int* cu_q, const int* slots, int n_entries, float* y_out,
                                     int H, int G, int N, int P, int taps, cudaStream_t stream) {
  if (n_entries <= 0) return ST_OK;
  if (int r = space_ok("state_space_walk", H, G, N, P, ldp, state_stride, n_entries)) return r;
  const int inner = H * P, C = inner + 2 * G * N;
  const long long carry = (long long)H * N * P;
  if (taps < 1 || state_stride < carry + (long long)C * (taps - 1))
    return refuse(ST_BAD_SIZE, "state_space_walk: taps=%d row=%lld", taps, state_stride);
  const int rpl = rows_per_lane(N);
  int cols = rpl <= 32 ? 64 : 32;
  if (cols > P) cols = (P + 3) / 4 * 4;
  const int vec = N % 4 == 0 && state_stride % 4 == 0 && ((uintptr_t)state & 15) == 0;
  const size_t smem = (2 * (size_t)rpl * kStateLanes + cols) * sizeof(float);
  ConvInput in{proj + inner, ldp, nullptr, state, state_stride, (int)carry, taps, C};
  const SpaceSizes z{H, G, N, P};
  dim3 grid((P + cols - 1) / cols, H, n_entries);
#define SRLM_SSW(R)                                                                                                       \
  launch_pdl(state_space_walk_kernel<R>, grid, dim3(cols * kStateLanes), smem, stream, in, conv_w, conv_b, proj + inner + C, \
             dt_bias, a_log, D, state, cu_q, slots, y_out, z, cols, vec)
  if (rpl == 4) SRLM_SSW(4);
  else if (rpl == 8) SRLM_SSW(8);
  else if (rpl == 16) SRLM_SSW(16);
  else if (rpl == 32) SRLM_SSW(32);
  else SRLM_SSW(64);
#undef SRLM_SSW
  return launched();
}

// Floats of a group's record for one head (0: heads of these sizes go token by token).
extern "C" int srlm_state_space_record(int N) { return N > 0 && N <= 256 ? kSpaceRecord : 0; }

// groups: how many groups of 8 tokens the step's entries have together; records float32 [groups, H, record]; conv float32
// [T, H P + 2 G N].
extern "C" int srlm_state_space_groups(const float* conv, const float* proj, long long ldp, const float* dt_bias,
                                       const float* a_log, const int* cu_q, int n_entries, float* records, int groups, int H,
                                       int G, int N, int P, cudaStream_t stream) {
  if (n_entries <= 0 || groups <= 0) return ST_OK;
  if (int r = space_ok("state_space_groups", H, G, N, P, ldp, 0x7fffffffffffLL, n_entries)) return r;
  const int inner = H * P, C = inner + 2 * G * N;
  launch_pdl(state_space_groups_kernel, dim3(groups, (H + 3) / 4), dim3(128), 0, stream, conv, C, proj + inner + C, ldp, dt_bias,
             a_log, cu_q, n_entries, records, SpaceSizes{H, G, N, P});
  return launched();
}

// The walk along the records that srlm_state_space_groups made; y_out float32 [T, H P].
extern "C" int srlm_state_space_read(const float* records, const float* conv, const float* D, float* state,
                                     long long state_stride, const int* cu_q, const int* slots, int n_entries, float* y_out,
                                     int H, int G, int N, int P, cudaStream_t stream) {
  if (n_entries <= 0) return ST_OK;
  if (int r = space_ok("state_space_read", H, G, N, P, 0x7fffffffffffLL, state_stride, n_entries)) return r;
  if (N > 256) return refuse(ST_BAD_SIZE, "state_space_read: state=%d (at most 256)", N);
  if (((uintptr_t)records & 15) != 0) return refuse(ST_BAD_ALIGN, "state_space_read: records must be 16-byte aligned");
  const int inner = H * P, C = inner + 2 * G * N, rpl = rows_per_lane(N);
  const SpaceSizes z{H, G, N, P};
  const int vec = N % 4 == 0 && state_stride % 4 == 0 && ((uintptr_t)state & 15) == 0;
  const int vec_rows = N % 4 == 0 && inner % 4 == 0 && ((uintptr_t)conv & 15) == 0;
  const size_t smem = (size_t)kSpaceStages * (2 * kStateGroup * rpl * kStateLanes + kSpaceRecord + kStateGroup * kSpaceCols) *
                      sizeof(float);
  dim3 grid((P + kSpaceCols - 1) / kSpaceCols, H, n_entries);
#define SRLM_SSR(ROWS, L)                                                                                               \
  do {                                                                                                                  \
    auto kern = state_space_read_kernel<ROWS, L>;                                                                       \
    if (smem > 40 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);           \
    launch_pdl_if(false, kern, grid, dim3(kSpaceThreads), smem, stream, records, conv, C, D, state, state_stride, cu_q, slots, \
                  y_out, z, vec, vec_rows);                                                                             \
  } while (0)
  if (rpl == 4) SRLM_SSR(32, 8);
  else if (rpl == 8) SRLM_SSR(64, 16);
  else if (rpl == 16) SRLM_SSR(128, 32);
  else SRLM_SSR(256, 32);
#undef SRLM_SSR
  return launched();
}

// y float32 [T, inner]; z: the first inner columns of proj; w float32 [inner]; parts: equal parts that are normed apart.
extern "C" int srlm_state_space_output(const float* y, const float* proj, long long ldp, const float* w, float eps, void* out,
                                       int out_dtype, int T, int inner, int parts, cudaStream_t stream) {
  if (T <= 0) return ST_OK;
  if (inner <= 0 || parts <= 0 || inner % parts || parts > 65535 || ldp < inner || !(eps > 0.f) || T > 65535 ||
      inner / parts > 12000)
    return refuse(ST_BAD_SIZE, "state_space_output: inner=%d parts=%d T=%d ld=%lld", inner, parts, T, ldp);
  const int part = inner / parts;
  int block = 32;
  while (block < 512 && block * 4 < part) block <<= 1;
  SRLM_DISPATCH_ACT(out_dtype, TO, launch_pdl(state_space_output_kernel<TO>, dim3(parts, T), dim3(block), part * sizeof(float),
                                              stream, y, proj, ldp, w, eps, (TO*)out, inner, part));
  return launched();
}
