// The gated delta rule with a decay per head AND key channel, on one matrix of state S [dk, dv] per head and request:
//
//   S <- diag(g) S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q            (in this order, per token)
//
// with q and k unit vectors per head (q also times dk^-1/2), both and v behind a short causal convolution over time and
// silu, beta = logistic(b), g = exp(-exp(A_h) softplus(a + dt)), one number a head and key channel.  Then per head
// o / rms(o) * w * logistic(gate).  Everything behind the projections is float32.
//
// proj float32 [T, ldp]: q (G dk) | k (G dk) | v (H dv) | b (H) | ...;  low float32 [T, ldl]: a (H dk) | gate (H dv).
// A request's state row: S [H][dv][dk] (a column of S contiguous) | the last taps - 1 inputs of the q, k and v channels
// ([taps - 1][channels], renewed by conv_carry behind the kernels that read them).
//
// Steps of short portions (decoding) take channel_delta_walk: one launch does convolution, decays, recurrence and, where a
// block holds a whole head, norm, gate and rounding; any sizes.  Steps with longer portions go by groups of 8 tokens:
//   channel_delta_groups   what 8 tokens do to a column of S and of v, which all columns share.  With P_i = g_1 .. g_i
//                          (products within the group, elementwise) and R_j = g_(j+1) .. g_8:
//                             N_ij = sum_r k_i k_j g_(j+1) .. g_i (j < i),  M_ij = likewise with q_i (j <= i),
//                             X = (I + diag(beta) N)^-1 diag(beta):  u = X (v - [P_i k_i . S]),  o_i = P_i q_i . S + (M u)_i
//                          and, with the products by X and M taken ahead of S,
//                             kx = X [P_i k_i],  qm = [P_i q_i] - M kx,  ke_j = R_j k_j,  whole = P_8,  MX = M X
//   channel_delta_read     walks the groups with S in registers, two products with S and one update a group:
//                             u = X v - kx . S,   o = MX v + qm . S,   S <- whole S + sum_j ke_j u_j
// The products of the decays never exceed 1, so nothing grows; a decay that underflows is a zero that stays one.
#include "state_walk.cuh"

namespace srlm {

struct DeltaSizes {
  int H, G, dk, dv;
};

// ---- token by token ----------------------------------------------------------------------------------------------------
// Block: `cols` columns (8 lanes each) of one head's S for one entry.
template <int RPL, typename TO>
__global__ void __launch_bounds__(RPL <= 16 ? 1024 : RPL <= 32 ? 512 : 256)
channel_delta_walk_kernel(ConvInput in, const float* __restrict__ conv_w, const float* __restrict__ low, long long ldl,
                          const float* __restrict__ a_log, const float* __restrict__ dt_bias, float* __restrict__ state,
                          const int* __restrict__ cu_q, const int* __restrict__ slots, const float* __restrict__ norm_w,
                          float eps, float* __restrict__ o_out, TO* __restrict__ out, DeltaSizes z, int cols, float unit_eps,
                          int vec) {
  constexpr int DKP = RPL * kStateLanes;
  extern __shared__ __align__(16) float walk_smem[];
  float* k_s = walk_smem;                    // [DKP] each, zeros behind dk
  float* q_s = k_s + DKP;
  float* g_s = q_s + DKP;
  float* v_s = g_s + DKP;                    // [cols]
  float* o_s = v_s + cols;                   // [cols]
  __shared__ float scalars[4];               // 1 / |k|, 1 / |q|, q . k, beta
  __shared__ float scratch[32];
  const int e = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * cols;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int cg = tid / kStateLanes, l = tid % kStateLanes, col = c0 + cg;
  const bool live = col < z.dv;
  const int kh = h / (z.H / z.G), width = min(cols, z.dv - c0);
  const int slot = slots[e];
  float* S_col = state + (size_t)slot * in.state_stride + ((size_t)h * z.dv + (live ? col : 0)) * z.dk;
  float S[RPL];
  pdl_wait();                                // what the kernels ahead wrote is read from here on
  pdl_trigger();
  load_column<RPL>(S, S_col, l, z.dk, live, vec);
  const float rate = expf(a_log[h]);
  const int t0 = cu_q[e], n = cu_q[e + 1] - t0;
  for (int i = tid; i < 3 * DKP; i += blockDim.x) walk_smem[i] = 0.f;
  for (int i = 0; i < n; ++i) {
    const int t = t0 + i;
    __syncthreads();                         // the token before is no longer read
    for (int x = tid; x < 2 * z.dk + width; x += blockDim.x) {
      const int part = x / z.dk;
      const int c = part == 0 ? (z.G + kh) * z.dk + x : part == 1 ? kh * z.dk + (x - z.dk)
                                                      : 2 * z.G * z.dk + h * z.dv + c0 + (x - 2 * z.dk);
      const float y = silu_of(conv_at(in, conv_w, t, i, slot, c));
      (part == 0 ? k_s + x : part == 1 ? q_s + (x - z.dk) : v_s + (x - 2 * z.dk))[0] = y;
    }
    for (int r = tid; r < z.dk; r += blockDim.x) {
      const float a = low[(size_t)t * ldl + (size_t)h * z.dk + r] + dt_bias[(size_t)h * z.dk + r];
      g_s[r] = expf(-rate * softplus_f(a));
    }
    __syncthreads();
    if (warp < 3) {                          // the block has four warps or more
      const float* x = warp == 1 ? q_s : k_s;
      const float* y = warp == 0 ? k_s : q_s;
      float ss = 0.f;
      for (int r = lane; r < z.dk; r += 32) ss += x[r] * y[r];
      ss = warp_sum(ss);
      if (lane == 0) scalars[warp] = warp == 2 ? ss : 1.f / sqrtf(ss + unit_eps);
    } else if (warp == 3 && lane == 0) {
      const float b = in.proj[(size_t)t * in.ld + in.C + h];
      scalars[3] = logistic_f(b);
    }
    __syncthreads();
    const float kn = scalars[0], qn = scalars[1] / sqrtf((float)z.dk), beta = scalars[3];
    float2 a2 = make_float2(0.f, 0.f), b2 = make_float2(0.f, 0.f);
#pragma unroll
    for (int j = 0; j < RPL / 4; ++j) {
      const float4 kv = *reinterpret_cast<const float4*>(k_s + 32 * j + 4 * l);
      const float4 qv = *reinterpret_cast<const float4*>(q_s + 32 * j + 4 * l);
      const float4 gv = *reinterpret_cast<const float4*>(g_s + 32 * j + 4 * l);
      S[4 * j] *= gv.x; S[4 * j + 1] *= gv.y; S[4 * j + 2] *= gv.z; S[4 * j + 3] *= gv.w;
      const float2 s0 = make_float2(S[4 * j], S[4 * j + 1]), s1 = make_float2(S[4 * j + 2], S[4 * j + 3]);
      a2 = fma2(make_float2(kv.x, kv.y), s0, a2);
      a2 = fma2(make_float2(kv.z, kv.w), s1, a2);
      b2 = fma2(make_float2(qv.x, qv.y), s0, b2);
      b2 = fma2(make_float2(qv.z, qv.w), s1, b2);
    }
    float a = a2.x + a2.y, b = b2.x + b2.y;
#pragma unroll
    for (int o = 1; o < kStateLanes; o <<= 1) {
      a += __shfl_xor_sync(0xffffffffu, a, o);
      b += __shfl_xor_sync(0xffffffffu, b, o);
    }
    const float u = live ? beta * (v_s[cg] - kn * a) : 0.f;
    const float o = qn * (b + scalars[2] * kn * u);
    const float ku = kn * u;
#pragma unroll
    for (int j = 0; j < RPL / 4; ++j) {
      const float4 kv = *reinterpret_cast<const float4*>(k_s + 32 * j + 4 * l);
      S[4 * j] = fmaf(kv.x, ku, S[4 * j]);
      S[4 * j + 1] = fmaf(kv.y, ku, S[4 * j + 1]);
      S[4 * j + 2] = fmaf(kv.z, ku, S[4 * j + 2]);
      S[4 * j + 3] = fmaf(kv.w, ku, S[4 * j + 3]);
    }
    if (o_out) {
      if (live && l == 0) o_out[((size_t)t * z.H + h) * z.dv + col] = o;
    } else {                                 // the block holds the whole head: norm, gate, rounding
      if (l == 0) o_s[cg] = live ? o : 0.f;
      const float inv = 1.f / sqrtf(block_sum(l == 0 && live ? o * o : 0.f, scratch) / (float)z.dv + eps);
      for (int c = tid; c < width; c += blockDim.x) {
        const float gate = low[(size_t)t * ldl + (size_t)z.H * z.dk + (size_t)h * z.dv + c];
        out[((size_t)t * z.H + h) * z.dv + c] = from_float<TO>(o_s[c] * inv * norm_w[c] * logistic_f(gate));
      }
    }
  }
  store_column<RPL>(S, S_col, l, z.dk, live, vec);
}

// ---- groups of 8 tokens ------------------------------------------------------------------------------------------------
// A group's record for one head, floats: kx [8][dkp] | qm [8][dkp] | ke [8][dkp] | whole [dkp] | X [8][8] | MX [8][8].
__host__ __device__ inline int delta_record(int dkp) { return 25 * dkp + 2 * kStateGroup * kStateGroup; }

// A block per (group, head), R key channels a thread.  conv: the convolved and activated q | k | v channels, float32 [T, C].
template <int R>
__global__ void __launch_bounds__(128)
channel_delta_groups_kernel(const float* __restrict__ conv, int C, const float* __restrict__ proj, long long ldp,
                            const float* __restrict__ low, long long ldl, const float* __restrict__ a_log,
                            const float* __restrict__ dt_bias, const int* __restrict__ cu_q, int n_entries,
                            float* __restrict__ records, DeltaSizes z, int dkp, float unit_eps) {
  pdl_wait();
  pdl_trigger();
  constexpr int M = kStateGroup;
  __shared__ float unit_s[2 * M];            // 1 / |k_i|, then dk^-1/2 / |q_i|
  __shared__ float beta_s[M];
  __shared__ float part[4][64];
  __shared__ float coef[64];
  __shared__ __align__(16) float x_s[M][M], m_s[M][M];
  const GroupHome home = group_home(cu_q, n_entries, blockIdx.x);
  if (home.entry < 0) return;
  const int h = blockIdx.y, kh = h / (z.H / z.G), tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  float k[R][M], q[R][M], g[R][M], sums[2 * M];
#pragma unroll
  for (int s = 0; s < 2 * M; ++s) sums[s] = 0.f;
#pragma unroll
  for (int x = 0; x < R; ++x) {
    const int r = tid + 128 * x;
    const float* row = conv + (size_t)home.t0 * C + (size_t)kh * z.dk + r;
    const float* a = low + (size_t)home.t0 * ldl + (size_t)h * z.dk + r;
#pragma unroll
    for (int i = 0; i < M; ++i) {
      const bool there = i < home.n && r < z.dk;
      q[x][i] = there ? row[(size_t)i * C] : 0.f;
      k[x][i] = there ? row[(size_t)i * C + (size_t)z.G * z.dk] : 0.f;
      g[x][i] = there ? a[(size_t)i * ldl] : 0.f;
    }
  }
  if (tid < M) beta_s[tid] = tid < home.n ? logistic_f(proj[(size_t)(home.t0 + tid) * ldp + C + h]) : 0.f;
  const float rate = expf(a_log[h]);
#pragma unroll
  for (int x = 0; x < R; ++x) {
    const int r = tid + 128 * x;
    const float bias = r < z.dk ? dt_bias[(size_t)h * z.dk + r] : 0.f;
#pragma unroll
    for (int i = 0; i < M; ++i) {
      sums[i] = fmaf(k[x][i], k[x][i], sums[i]);
      sums[M + i] = fmaf(q[x][i], q[x][i], sums[M + i]);
      g[x][i] = i < home.n && r < z.dk ? expf(-rate * softplus_f(g[x][i] + bias)) : 1.f;
    }
  }
  scatter_sums<2 * M, 2 * M>(sums, lane & 15);
  sums[0] += __shfl_xor_sync(0xffffffffu, sums[0], 16);
  if (lane < 2 * M) part[warp][lane] = sums[0];
  __syncthreads();
  if (tid < 2 * M)
    unit_s[tid] = (tid < M ? 1.f : 1.f / sqrtf((float)z.dk)) /
                  sqrtf((part[0][tid] + part[1][tid]) + (part[2][tid] + part[3][tid]) + unit_eps);
  __syncthreads();
  float* rec = records + ((size_t)blockIdx.x * z.H + h) * delta_record(dkp);
  float acc[64];                             // M_ij at i (i + 1) / 2 + j, N_ij at 36 + i (i - 1) / 2 + j
#pragma unroll
  for (int s = 0; s < 64; ++s) acc[s] = 0.f;
#pragma unroll
  for (int x = 0; x < R; ++x) {
    const int r = tid + 128 * x;
#pragma unroll
    for (int i = 0; i < M; ++i) {
      k[x][i] *= unit_s[i];
      q[x][i] *= unit_s[M + i];
    }
#pragma unroll
    for (int j = 0; j < M; ++j) {
      float f = k[x][j];
      acc[j * (j + 1) / 2 + j] += q[x][j] * f;
#pragma unroll
      for (int i = j + 1; i < M; ++i) {
        f *= g[x][i];
        acc[i * (i + 1) / 2 + j] += q[x][i] * f;
        acc[36 + i * (i - 1) / 2 + j] += k[x][i] * f;
      }
    }
  }
  scatter_sums<64, 32>(acc, lane);
  __syncthreads();                           // part is read
  part[warp][2 * lane] = acc[0];
  part[warp][2 * lane + 1] = acc[1];
  __syncthreads();
  if (tid < 64) coef[tid] = (part[0][tid] + part[1][tid]) + (part[2][tid] + part[3][tid]);
  __syncthreads();
  if (tid < M) {                             // column tid of X, forward along the rows
    float x[M];
#pragma unroll
    for (int i = 0; i < M; ++i) {
      float s = i == tid ? 1.f : 0.f;
#pragma unroll
      for (int j = 0; j < i; ++j) s -= coef[36 + i * (i - 1) / 2 + j] * x[j];
      x[i] = beta_s[i] * s;
      x_s[i][tid] = x[i];
    }
  } else if (tid >= 64) {
    const int i = (tid - 64) / M, j = (tid - 64) % M;
    m_s[i][j] = j <= i ? coef[i * (i + 1) / 2 + j] : 0.f;
  }
  __syncthreads();
  if (tid < M * M) {
    const int i = tid / M, j = tid % M;
    float s = 0.f;
    for (int y = 0; y <= i; ++y) s = fmaf(m_s[i][y], x_s[y][j], s);
    rec[25 * dkp + tid] = x_s[i][j];
    rec[25 * dkp + M * M + tid] = s;
  }
#pragma unroll
  for (int x = 0; x < R; ++x) {
    const int r = tid + 128 * x;
    if (r >= dkp) break;
    float pre = 1.f, suf = 1.f;
#pragma unroll
    for (int i = M - 1; i >= 0; --i) {
      rec[(2 * M + i) * dkp + r] = k[x][i] * suf;
      suf *= g[x][i];
    }
#pragma unroll
    for (int i = 0; i < M; ++i) {
      pre *= g[x][i];
      k[x][i] *= pre;
      q[x][i] *= pre;
    }
    rec[3 * M * dkp + r] = pre;
    float kx[M];
#pragma unroll
    for (int i = 0; i < M; ++i) {
      float s = 0.f, qm = q[x][i];
#pragma unroll
      for (int j = 0; j <= i; ++j) s = fmaf(x_s[i][j], k[x][j], s);
      kx[i] = s;
#pragma unroll
      for (int j = 0; j <= i; ++j) qm = fmaf(-m_s[i][j], kx[j], qm);
      rec[i * dkp + r] = s;
      rec[(M + i) * dkp + r] = qm;
    }
  }
}

// Block: 16 columns of one head's S for one entry, four a warp; a group's record comes into one of three stages while the
// two ahead of it are worked on.
constexpr int kReadCols = 16, kReadStages = 3, kReadThreads = 128;      // 128 = 8 tokens x 16 columns: a value a thread

template <int DKP, int L>
__global__ void __launch_bounds__(kReadThreads, 2)      // two blocks an SM: registers for many loads in flight
channel_delta_read_kernel(const float* __restrict__ records, const float* __restrict__ conv, int C, float* __restrict__ state,
                          long long state_stride, const int* __restrict__ cu_q, const int* __restrict__ slots,
                          float* __restrict__ o_out, DeltaSizes z, int vec) {
  pdl_wait();
  pdl_trigger();
  typedef StateTile<DKP, L> Tile;
  constexpr int M = kStateGroup, REC = 25 * DKP + 2 * M * M, NC = Tile::kColumns;
  constexpr int STAGE = REC + M * kReadCols;
  extern __shared__ __align__(16) float read_smem[];        // [kReadStages]: the record | v [8][16]
  __shared__ __align__(16) float u_s[kReadThreads / 32][32 * NC];
  const int e = blockIdx.z, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int hl = lane % L, set = lane / L, l = lane & 7;
  const int col_set = blockIdx.x * kReadCols + 4 * warp + set * NC;        // the first column that the lane holds rows of
  const int col = blockIdx.x * kReadCols + 4 * warp + (lane >> 3);         // the column whose token l the lane finishes
  const bool live = col < z.dv;
  const int t0 = cu_q[e], n = cu_q[e + 1] - t0, groups = (n + M - 1) / M;
  const float* rec0 = records + ((size_t)first_group(cu_q, e) * z.H + h) * REC;
  const int v_col = blockIdx.x * kReadCols + tid % kReadCols;
  const float* v_in = conv + 2 * (size_t)z.G * z.dk + (size_t)h * z.dv + v_col;
  auto fetch = [&](int g) {
    if (g < groups) {
      const float* src = rec0 + (size_t)g * z.H * REC;
      float* dst = read_smem + (g % kReadStages) * STAGE;
#pragma unroll
      for (int i = tid * 4; i < REC; i += kReadThreads * 4) state_copy_16(dst + i, src + i);
      const int tok = g * M + tid / kReadCols;              // a thread's value of the group
      if (tok < n && v_col < z.dv) state_copy_4(dst + REC + tid, v_in + (size_t)(t0 + tok) * C);
      else dst[REC + tid] = 0.f;
    }
    state_copy_commit();
  };
  fetch(0);
  fetch(1);
  float* S_head = state + (size_t)slots[e] * state_stride + (size_t)h * z.dv * z.dk;
  Tile S;
  S.load(S_head, col_set, z.dv, hl, z.dk, vec);
  int row_of[M];                             // where the lane's piece of the vector of token slot i lies
#pragma unroll
  for (int i = 0; i < M; ++i) row_of[i] = (i ^ l) * DKP + 4 * hl;
  for (int g = 0; g < groups; ++g) {
    state_copy_wait<1>();
    __syncthreads();                         // group g is here for all; group g - 1 is read by all
    fetch(g + 2);
    const float* st = read_smem + (g % kReadStages) * STAGE;
    float p[8 * NC], w[8 * NC];              // slots of column c and token i, at 8 c + i: kx_i . S, then qm_i . S
#pragma unroll
    for (int i = 0; i < M; ++i) {
      float a[NC];
      S.dot(st + row_of[i], a);
#pragma unroll
      for (int c = 0; c < NC; ++c) p[8 * c + i] = a[c];
    }
    const float4* X = reinterpret_cast<const float4*>(st + 25 * DKP + l * M);
    const float4 x0 = X[0], x1 = X[1], m0 = X[M * M / 4], m1 = X[M * M / 4 + 1];
    const float xr[M] = {x0.x, x0.y, x0.z, x0.w, x1.x, x1.y, x1.z, x1.w};
    const float mr[M] = {m0.x, m0.y, m0.z, m0.w, m1.x, m1.y, m1.z, m1.w};
    float u = 0.f, o = 0.f;
#pragma unroll
    for (int j = 0; j < M; ++j) {
      const float v = st[REC + j * kReadCols + 4 * warp + (lane >> 3)];
      u = fmaf(xr[j], v, u);
      o = fmaf(mr[j], v, o);
    }
    permuted_sums<8 * NC, L>(p);
    u -= p[0];
    Tile::share(u_s[warp], set, hl, u);
#pragma unroll
    for (int i = 0; i < M; ++i) {            // does not wait for u: fills the exchanges' latency
      float a[NC];
      S.dot(st + M * DKP + row_of[i], a);
#pragma unroll
      for (int c = 0; c < NC; ++c) w[8 * c + i] = a[c];
    }
#pragma unroll
    for (int j = 0; j < Tile::kPieces; ++j) {
      const float4 wh = *reinterpret_cast<const float4*>(st + 3 * M * DKP + 4 * hl + 4 * L * j);
#pragma unroll
      for (int c = 0; c < NC; ++c) {
        S.s[c][2 * j].x *= wh.x; S.s[c][2 * j].y *= wh.y;
        S.s[c][2 * j + 1].x *= wh.z; S.s[c][2 * j + 1].y *= wh.w;
      }
    }
    __syncwarp();
#pragma unroll
    for (int j = 0; j < M; ++j) {
      alignas(16) float uj[NC];
      Tile::shared(u_s[warp], set, hl, j, uj);
      S.add(st + (2 * M + j) * DKP + 4 * hl, uj);
    }
    permuted_sums<8 * NC, L>(w);
    o += w[0];
    if (live && g * M + l < n) o_out[((size_t)(t0 + g * M + l) * z.H + h) * z.dv + col] = o;
  }
  state_copy_wait<0>();
  S.store(S_head, col_set, z.dv, hl, z.dk, vec);
}

}  // namespace srlm

using namespace srlm;

static int channel_delta_ok(const char* what, int H, int G, int dk, int dv, int n_entries) {
  if (H <= 0 || G <= 0 || H % G || dk <= 0 || dk > 512 || dv <= 0 || H > 65535 || n_entries > 65535)
    return refuse(ST_BAD_SIZE, "%s: H=%d G=%d dk=%d (at most 512) dv=%d entries=%d", what, H, G, dk, dv, n_entries);
  return ST_OK;
}
static int rows_per_lane(int rows) { return rows <= 32 ? 4 : rows <= 64 ? 8 : rows <= 128 ? 16 : rows <= 256 ? 32 : 64; }
static int walk_columns(int rpl) { return rpl <= 16 ? 128 : rpl <= 32 ? 64 : 32; }

// Whether channel_delta_walk norms and gates itself (one tile of columns holds a head).
extern "C" int srlm_channel_delta_walk_finishes(int dk, int dv) { return dv <= walk_columns(rows_per_lane(dk)); }

// conv_w float32 [C, taps] stacked as the channels; norm_w float32 [dv]; state float32 [slots, state_stride]; out [T, H dv]
// where the walk finishes (srlm_channel_delta_walk_finishes), else o_out float32 [T, H dv].
extern "C" int srlm_channel_delta_walk(const float* proj, long long ldp, const float* conv_w, const float* low, long long ldl,
                                       const float* a_log, const float* dt_bias, float* state, long long state_stride,
                                       const int* cu_q, const int* slots, int n_entries, const float* norm_w, float eps,
                                       float* o_out, void* out, int out_dtype, int H, int G, int dk, int dv, int taps,
                                       float unit_eps, cudaStream_t stream) {
  if (n_entries <= 0) return ST_OK;
  if (int r = channel_delta_ok("channel_delta_walk", H, G, dk, dv, n_entries)) return r;
  const int C = 2 * G * dk + H * dv;
  const long long carry = (long long)H * dk * dv;
  if (taps < 1 || ldp < C + H || ldl < (long long)H * (dk + dv) || state_stride < carry + (long long)C * (taps - 1) ||
      carry > 0x7fffffffLL || !(eps > 0.f))
    return refuse(ST_BAD_SIZE, "channel_delta_walk: taps=%d ldp=%lld ldl=%lld state=%lld", taps, ldp, ldl, state_stride);
  const bool finishes = srlm_channel_delta_walk_finishes(dk, dv);
  if (finishes ? !out : !o_out) return refuse(ST_BAD_SIZE, "channel_delta_walk: no buffer for the result");
  const int rpl = rows_per_lane(dk);
  int cols = walk_columns(rpl);
  if (cols > dv) cols = (dv + 3) / 4 * 4;
  if (cols < 16) cols = 16;                                // four warps at least
  const int vec = dk % 4 == 0 && state_stride % 4 == 0 && ((uintptr_t)state & 15) == 0;
  const size_t smem = (3 * (size_t)rpl * kStateLanes + 2 * cols) * sizeof(float);
  ConvInput in{proj, ldp, nullptr, state, state_stride, (int)carry, taps, C};
  const DeltaSizes z{H, G, dk, dv};
  dim3 grid((dv + cols - 1) / cols, H, n_entries);
#define SRLM_CDW(R)                                                                                                        \
  SRLM_DISPATCH_ACT(out_dtype, TO, launch_pdl(channel_delta_walk_kernel<R, TO>, grid, dim3(cols * kStateLanes), smem, stream, \
      in, conv_w, low, ldl, a_log, dt_bias, state, cu_q, slots, norm_w, eps, finishes ? (float*)nullptr : o_out, (TO*)out, z,  \
      cols, unit_eps, vec))
  if (rpl == 4) SRLM_CDW(4);
  else if (rpl == 8) SRLM_CDW(8);
  else if (rpl == 16) SRLM_CDW(16);
  else if (rpl == 32) SRLM_CDW(32);
  else SRLM_CDW(64);
#undef SRLM_CDW
  return launched();
}

// Whether steps may go by groups of tokens, and how many floats a group's record takes for one head (0: they may not).
extern "C" int srlm_channel_delta_record(int dk) { return dk > 0 && dk <= 256 ? delta_record(rows_per_lane(dk) * kStateLanes) : 0; }

// groups: how many groups of 8 tokens the step's entries have together; records float32 [groups, H, record]; conv float32
// [T, C].
extern "C" int srlm_channel_delta_groups(const float* conv, const float* proj, long long ldp, const float* low, long long ldl,
                                         const float* a_log, const float* dt_bias, const int* cu_q, int n_entries,
                                         float* records, int groups, int H, int G, int dk, int dv, float unit_eps,
                                         cudaStream_t stream) {
  if (n_entries <= 0 || groups <= 0) return ST_OK;
  if (int r = channel_delta_ok("channel_delta_groups", H, G, dk, dv, n_entries)) return r;
  const int C = 2 * G * dk + H * dv;
  if (!srlm_channel_delta_record(dk) || ldp < C + H || ldl < (long long)H * dk)
    return refuse(ST_BAD_SIZE, "channel_delta_groups: dk=%d (at most 256) ldp=%lld ldl=%lld", dk, ldp, ldl);
  const int dkp = rows_per_lane(dk) * kStateLanes;
  auto kern = dkp <= 128 ? channel_delta_groups_kernel<1> : channel_delta_groups_kernel<2>;
  launch_pdl(kern, dim3(groups, H), dim3(128), 0, stream, conv, C, proj, ldp, low, ldl, a_log, dt_bias, cu_q, n_entries, records,
             DeltaSizes{H, G, dk, dv}, dkp, unit_eps);
  return launched();
}

// The walk along the records that srlm_channel_delta_groups made; o_out float32 [T, H dv].
extern "C" int srlm_channel_delta_read(const float* records, const float* conv, float* state, long long state_stride,
                                       const int* cu_q, const int* slots, int n_entries, float* o_out, int H, int G, int dk,
                                       int dv, cudaStream_t stream) {
  if (n_entries <= 0) return ST_OK;
  if (int r = channel_delta_ok("channel_delta_read", H, G, dk, dv, n_entries)) return r;
  if (!srlm_channel_delta_record(dk) || state_stride < (long long)H * dk * dv)
    return refuse(ST_BAD_SIZE, "channel_delta_read: dk=%d (at most 256) state=%lld", dk, state_stride);
  if (((uintptr_t)records & 15) != 0) return refuse(ST_BAD_ALIGN, "channel_delta_read: records must be 16-byte aligned");
  const int C = 2 * G * dk + H * dv, rpl = rows_per_lane(dk);
  const DeltaSizes z{H, G, dk, dv};
  const int vec = dk % 4 == 0 && state_stride % 4 == 0 && ((uintptr_t)state & 15) == 0;
  const size_t smem = (size_t)kReadStages * (delta_record(rpl * kStateLanes) + kStateGroup * kReadCols) * sizeof(float);
  dim3 grid((dv + kReadCols - 1) / kReadCols, H, n_entries);
#define SRLM_CDR(ROWS, L)                                                                                               \
  do {                                                                                                                  \
    auto kern = channel_delta_read_kernel<ROWS, L>;                                                                     \
    if (smem > 40 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);           \
    launch_pdl_if(false, kern, grid, dim3(kReadThreads), smem, stream, records, conv, C, state, state_stride, cu_q, slots, \
                  o_out, z, vec);                                                                                       \
  } while (0)
  if (rpl == 4) SRLM_CDR(32, 8);
  else if (rpl == 8) SRLM_CDR(64, 16);
  else if (rpl == 16) SRLM_CDR(128, 32);
  else SRLM_CDR(256, 32);
#undef SRLM_CDR
  return launched();
}
