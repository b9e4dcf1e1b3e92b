// The gated delta rule: a recurrence that writes the difference between a value and what its key already reads.
// float32 arithmetic and state; the element type of the projections (float or bfloat16) is a template parameter.
//
// Per request and head, with the q and k of group h / (heads / groups), each divided by sqrt(sum of squares + unit_eps), q
// also times q_scale:
//     g_t = exp(-exp(a_log[h]) softplus(a_t + dt_bias[h])),   beta_t = sigmoid(b_t)
//     S <- g_t S,   u_t = beta_t (v_t - S^T k_t),   S <- S + k_t u_t^T,   o_t = S^T q_t
// S [dim, vdim] starts at zero and lives in the request's state slot.
//
//  * delta_walk:     token by token, for single tokens and short portions.  One block per (request, head, block of value
//                    columns) with its part of S in registers.
//  * long portions in chunks of 64 tokens, four launches.  With G_i the sum of log g up to token i of a chunk and S_0
//    the state before it, the recurrence inside a chunk is a triangular system for the rows u_i:
//        u_i + sum_(j<i) A_ij u_j = beta_i v_i - beta_i e^(G_i) S_0^T k_i,    A_ij = beta_i e^(G_i - G_j) k_i . k_j
//    so U = U0 - W S_0 with (I + A) U0 = diag(beta) V and (I + A) W = diag(beta e^G) K, both independent of S_0:
//      delta_prepare:  per (chunk, head) the scores, U0 and W by forward substitution (a thread per column), and the
//                      decayed keys e^(G_last - G_j) k_j and queries e^(G_i) q_i;
//      delta_carry:    per (request, head, 16 value columns), chunk after chunk: U = U0 - W S, S <- e^(G_last) S + K~^T U;
//                      keeps U and the state before each chunk;
//      delta_outputs:  per (chunk, head, 64 columns) o_i = e^(G_i) S_0^T q_i + sum_(j<=i) e^(G_i - G_j) (q_i . k_j) u_j.
//    Differences of G are never positive where they are used, so no exponential overflows.
#include "common.cuh"

namespace {

constexpr int DELTA_CHUNK = 64;

__device__ __forceinline__ float dr_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float dr_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }

template <typename T>
struct DeltaParams {
  const T* q; const T* k; const T* v; int stride;          // rows [tokens, groups * dim | groups * dim | heads * vdim], one stride
  const T* b; const T* a; int gate_stride;                 // [tokens, heads] each, one stride
  const float* a_log; const float* dt_bias;                // [heads]
  int heads, groups, dim, vdim, requests;
  float q_scale, unit_eps;
  const int* q_start; const int* state_slots; float* state; int num_slots;
  float* out;                                              // [tokens, heads * vdim]
  int* status;
  // scratch of the chunked form, per (chunk, head): W, decayed keys and queries [64, dim_pad], U [64, v_pad], scores of the
  // queries [64, 64], the state before the chunk [dim_pad, v_pad], e^(G_last)
  int dim_pad, v_pad;
  float* w; float* kd; float* qd; float* u; float* scores; float* before; float* decay;
};

// ------------------------------------------------------------------------------------------ token by token
constexpr int WALK_THREADS = 128, WALK_ROWS = 8, WALK_COLS = 4, WALK_BATCH = 8;

// A thread holds 8 rows (slice, slice + slices, ...) x 4 columns of S; the `slices` lanes of a column group add their parts
// with shuffles.  Tokens are staged WALK_BATCH at a time, a warp per token: raw q and k beside their norms' factors, the
// decay, the write strength and q . k, so that one reduction per token serves both products with the old state:
// o = S_new^T q = g S^T q + (k . q) u.
template <typename T>
__global__ void __launch_bounds__(WALK_THREADS)
delta_walk_kernel(const DeltaParams<T> p, int slices_log2) {
  extern __shared__ float4 walk_smem[];
  const int slices = 1 << slices_log2, rows_pad = WALK_ROWS << slices_log2, cb = WALK_THREADS / slices * WALK_COLS;
  float2* qk = reinterpret_cast<float2*>(walk_smem);                                              // [WALK_BATCH][rows_pad]
  float* vt = reinterpret_cast<float*>(qk + WALK_BATCH * rows_pad);    // [WALK_BATCH][cb]
  float4* scalars = reinterpret_cast<float4*>(vt + WALK_BATCH * cb);   // [WALK_BATCH]: k's factor, q's factor, g, beta
  float* cross = reinterpret_cast<float*>(scalars + WALK_BATCH);       // [WALK_BATCH]: q . k of the unit vectors
  pdl_launch_dependents();
  pdl_wait();
  const int r = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int first = p.q_start[r], last = p.q_start[r + 1];
  if (first >= last) return;
  const int slot = p.state_slots[r];
  if (slot < 0 || slot >= p.num_slots) {
    if (tid == 0) atomicOr(p.status, SPROUT_STATUS_BAD_PAGE);
    return;
  }
  const int slice = tid & (slices - 1), col_local = (tid >> slices_log2) * WALK_COLS, col = blockIdx.z * cb + col_local;
  const int g = h / (p.heads / p.groups), dim = p.dim, vdim = p.vdim;
  float* mine = p.state + (((size_t)slot * p.heads + h) * dim) * vdim;
  const bool vectors = (vdim & 3) == 0;
  float S[WALK_ROWS][WALK_COLS];
#pragma unroll
  for (int j = 0; j < WALK_ROWS; j++) {
    const int row = j * slices + slice;
    if (vectors) {
      float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
      if (col < vdim && row < dim) x = *reinterpret_cast<const float4*>(mine + (size_t)row * vdim + col);
      S[j][0] = x.x; S[j][1] = x.y; S[j][2] = x.z; S[j][3] = x.w;
    } else {
#pragma unroll
      for (int c = 0; c < WALK_COLS; c++) S[j][c] = (col + c < vdim && row < dim) ? mine[(size_t)row * vdim + col + c] : 0.f;
    }
  }
  const float rate = expf(p.a_log[h]), bias = p.dt_bias[h];
  for (int t0 = first; t0 < last; t0 += WALK_BATCH) {
    const int n = min(WALK_BATCH, last - t0);
    __syncthreads();                                                   // the batch before has been read by everyone
    for (int tt = warp; tt < n; tt += WALK_THREADS / 32) {
      const size_t t = t0 + tt;
      const T* qrow = p.q + t * p.stride + (size_t)g * dim;
      const T* krow = p.k + t * p.stride + (size_t)g * dim;
      float qq = 0.f, kk = 0.f, qk_sum = 0.f;
      for (int i = lane; i < rows_pad; i += 32) {
        const float x = i < dim ? to_float(qrow[i]) : 0.f, y = i < dim ? to_float(krow[i]) : 0.f;
        qk[tt * rows_pad + i] = make_float2(x, y);
        qq = fmaf(x, x, qq);
        kk = fmaf(y, y, kk);
        qk_sum = fmaf(x, y, qk_sum);
      }
      for (int i = lane; i < cb; i += 32) {
        const int column = blockIdx.z * cb + i;
        vt[tt * cb + i] = column < vdim ? to_float(p.v[t * p.stride + (size_t)h * vdim + column]) : 0.f;
      }
      qq = warp_sum(qq);
      kk = warp_sum(kk);
      qk_sum = warp_sum(qk_sum);
      if (lane == 0) {
        const float fq = p.q_scale / sqrtf(qq + p.unit_eps), fk = 1.0f / sqrtf(kk + p.unit_eps);
        const float decay = expf(-rate * dr_softplus(to_float(p.a[t * p.gate_stride + h]) + bias));
        scalars[tt] = make_float4(fk, fq, decay, dr_sigmoid(to_float(p.b[t * p.gate_stride + h])));
        cross[tt] = qk_sum * fq * fk;
      }
    }
    __syncthreads();
    for (int tt = 0; tt < n; tt++) {
      const float4 sc = scalars[tt];
      const float kq = cross[tt];
      float k[WALK_ROWS], read[WALK_COLS], asked[WALK_COLS];
#pragma unroll
      for (int c = 0; c < WALK_COLS; c++) read[c] = asked[c] = 0.f;
#pragma unroll
      for (int j = 0; j < WALK_ROWS; j++) {
        const float2 x = qk[tt * rows_pad + j * slices + slice];
        const float q = x.x * sc.y;
        k[j] = x.y * sc.x;
#pragma unroll
        for (int c = 0; c < WALK_COLS; c++) {
          read[c] = fmaf(S[j][c], k[j], read[c]);
          asked[c] = fmaf(S[j][c], q, asked[c]);
        }
      }
      for (int d = slices >> 1; d > 0; d >>= 1) {
#pragma unroll
        for (int c = 0; c < WALK_COLS; c++) {
          read[c] += __shfl_xor_sync(0xffffffffu, read[c], d);
          asked[c] += __shfl_xor_sync(0xffffffffu, asked[c], d);
        }
      }
      float* dst = p.out + (size_t)(t0 + tt) * p.heads * vdim + (size_t)h * vdim + col;
#pragma unroll
      for (int c = 0; c < WALK_COLS; c++) {
        const float u = sc.w * (vt[tt * cb + col_local + c] - sc.z * read[c]);
#pragma unroll
        for (int j = 0; j < WALK_ROWS; j++) S[j][c] = fmaf(sc.z, S[j][c], k[j] * u);
        if (slice == 0 && col + c < vdim) dst[c] = fmaf(kq, u, sc.z * asked[c]);
      }
    }
  }
#pragma unroll
  for (int j = 0; j < WALK_ROWS; j++) {
    const int row = j * slices + slice;
    if (row >= dim) continue;
    if (vectors) {
      if (col < vdim) *reinterpret_cast<float4*>(mine + (size_t)row * vdim + col) = make_float4(S[j][0], S[j][1], S[j][2], S[j][3]);
    } else {
#pragma unroll
      for (int c = 0; c < WALK_COLS; c++)
        if (col + c < vdim) mine[(size_t)row * vdim + col + c] = S[j][c];
    }
  }
}

// ------------------------------------------------------------------------------------------ chunks
constexpr int DELTA_THREADS = 256, CARRY_COLS = 16, CARRY_STRIDE = CARRY_COLS + 4, OUT_COLS = 64;   // rows of 20 floats: no two of 8 lanes' rows share a bank
constexpr int PREP_A_STRIDE = DELTA_CHUNK + 4;

// The chunks of all requests are numbered in the requests' order, ceil(tokens / 64) each.
__device__ __forceinline__ bool delta_find_chunk(const int* q_start, int requests, int index, int& r, int& c) {
  for (int i = 0; i < requests; i++) {
    const int n = (q_start[i + 1] - q_start[i] + DELTA_CHUNK - 1) / DELTA_CHUNK;
    if (index < n) { r = i; c = index; return true; }
    index -= n;
  }
  return false;
}

__device__ __forceinline__ void dr_cp_async16(void* smem, const void* gmem) {
  const uint32_t dst = (uint32_t)__cvta_generic_to_shared(smem);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(gmem) : "memory");
}
__device__ __forceinline__ void dr_cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void dr_cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// x += a.b over four neighbours of both rows
__device__ __forceinline__ float dot4(const float4& a, const float4& b, float x) {
  return fmaf(a.w, b.w, fmaf(a.z, b.z, fmaf(a.y, b.y, fmaf(a.x, b.x, x))));
}

template <typename T>
__global__ void __launch_bounds__(DELTA_THREADS, 2)
delta_prepare_kernel(const DeltaParams<T> p) {
  extern __shared__ float4 prep_smem[];
  const int dim = p.dim, dp = p.dim_pad, ds = dp + 4;
  float* kn = reinterpret_cast<float*>(prep_smem);        // [64][ds], unit keys
  float* qn = kn + DELTA_CHUNK * ds;                      // [64][ds], unit queries times q_scale
  float* at = qn + DELTA_CHUNK * ds;                      // [64][PREP_A_STRIDE]: at[j][i] = A_ij, zero for i <= j
  __shared__ float s_beta[DELTA_CHUNK], s_g[DELTA_CHUNK], s_up[DELTA_CHUNK], s_down[DELTA_CHUNK];    // e^(G_i), e^(G_last - G_i)
  pdl_launch_dependents();
  pdl_wait();
  int r, c;
  if (!delta_find_chunk(p.q_start, p.requests, blockIdx.x, r, c)) return;
  const int h = blockIdx.y, g = h / (p.heads / p.groups), tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int first = p.q_start[r] + c * DELTA_CHUNK, n = min(DELTA_CHUNK, p.q_start[r + 1] - first);
  const size_t place = (size_t)blockIdx.x * p.heads + h;
  // unit keys and queries, a warp per token
  for (int i = warp; i < DELTA_CHUNK; i += DELTA_THREADS / 32) {
    const size_t t = first + i;
    const T* qrow = p.q + t * p.stride + (size_t)g * dim;
    const T* krow = p.k + t * p.stride + (size_t)g * dim;
    float qq = 0.f, kk = 0.f;
    for (int d = lane; d < dp; d += 32) {
      const float x = i < n && d < dim ? to_float(qrow[d]) : 0.f, y = i < n && d < dim ? to_float(krow[d]) : 0.f;
      qn[i * ds + d] = x;
      kn[i * ds + d] = y;
      qq = fmaf(x, x, qq);
      kk = fmaf(y, y, kk);
    }
    const float fq = p.q_scale / sqrtf(warp_sum(qq) + p.unit_eps), fk = 1.0f / sqrtf(warp_sum(kk) + p.unit_eps);
    for (int d = lane; d < dp; d += 32) {
      qn[i * ds + d] *= fq;
      kn[i * ds + d] *= fk;
    }
  }
  if (warp == 0) {
    // running sums of log g, in the tokens' order; tokens beyond the portion neither decay nor write
    const float rate = expf(p.a_log[h]), bias = p.dt_bias[h];
    float carried = 0.f;
#pragma unroll
    for (int half = 0; half < DELTA_CHUNK / 32; half++) {
      const int i = half * 32 + lane;
      const size_t t = first + i;
      float x = i < n ? -rate * dr_softplus(to_float(p.a[t * p.gate_stride + h]) + bias) : 0.f;
#pragma unroll
      for (int d = 1; d < 32; d <<= 1) {
        const float y = __shfl_up_sync(0xffffffffu, x, d);
        if (lane >= d) x += y;
      }
      x += carried;
      carried = __shfl_sync(0xffffffffu, x, 31);
      s_g[i] = x;
      s_up[i] = expf(x);
      s_beta[i] = i < n ? dr_sigmoid(to_float(p.b[t * p.gate_stride + h])) : 0.f;
    }
  }
  __syncthreads();
  {
    // k_i . k_j and q_i . k_j: thread (ti, tj) has rows ti + 16 a and columns tj + 16 b, blocks above the diagonal left out
    const int ti = tid >> 4, tj = tid & 15;
    float kk[4][4], qk[4][4];
#pragma unroll
    for (int a = 0; a < 4; a++)
#pragma unroll
      for (int b = 0; b < 4; b++) kk[a][b] = qk[a][b] = 0.f;
    for (int d = 0; d < dp; d += 4) {
      float4 kj[4];
#pragma unroll
      for (int b = 0; b < 4; b++) kj[b] = *reinterpret_cast<const float4*>(kn + (tj + 16 * b) * ds + d);
#pragma unroll
      for (int a = 0; a < 4; a++) {
        const float4 ki = *reinterpret_cast<const float4*>(kn + (ti + 16 * a) * ds + d);
        const float4 qi = *reinterpret_cast<const float4*>(qn + (ti + 16 * a) * ds + d);
#pragma unroll
        for (int b = 0; b <= a; b++) {
          kk[a][b] = dot4(ki, kj[b], kk[a][b]);
          qk[a][b] = dot4(qi, kj[b], qk[a][b]);
        }
      }
    }
    float* scores = p.scores + place * DELTA_CHUNK * DELTA_CHUNK;
#pragma unroll
    for (int a = 0; a < 4; a++)
#pragma unroll
      for (int b = 0; b < 4; b++) {
        const int i = ti + 16 * a, j = tj + 16 * b;
        const float fade = i >= j ? expf(s_g[i] - s_g[j]) : 0.f;
        at[j * PREP_A_STRIDE + i] = i > j ? s_beta[i] * fade * kk[a][b] : 0.f;
        scores[i * DELTA_CHUNK + j] = fade * qk[a][b];
      }
  }
  const float end = s_g[DELTA_CHUNK - 1];
  if (tid < DELTA_CHUNK) s_down[tid] = expf(end - s_g[tid]);
  __syncthreads();
  float* w = p.w + place * DELTA_CHUNK * dp;
  float* kd = p.kd + place * DELTA_CHUNK * dp;
  float* qd = p.qd + place * DELTA_CHUNK * dp;
  for (int e = tid; e < DELTA_CHUNK * dp; e += DELTA_THREADS) {
    const int i = e / dp, d = e % dp;
    kd[e] = kn[i * ds + d] * s_down[i];
    qd[e] = qn[i * ds + d] * s_up[i];
  }
  if (tid == 0) p.decay[place] = s_up[DELTA_CHUNK - 1];
  // forward substitution, a thread per column of [K | V]
  float* u = p.u + place * DELTA_CHUNK * p.v_pad;
  for (int column = tid; column < dp + p.v_pad; column += DELTA_THREADS) {
    float x[DELTA_CHUNK];
    if (column < dp) {
#pragma unroll
      for (int i = 0; i < DELTA_CHUNK; i++) x[i] = s_beta[i] * s_up[i] * kn[i * ds + column];
    } else {
      const int vc = column - dp;
      const T* src = p.v + (size_t)first * p.stride + (size_t)h * p.vdim + vc;
#pragma unroll
      for (int i = 0; i < DELTA_CHUNK; i++) x[i] = i < n && vc < p.vdim ? s_beta[i] * to_float(src[(size_t)i * p.stride]) : 0.f;
    }
#pragma unroll
    for (int j = 0; j < DELTA_CHUNK - 1; j++) {
#pragma unroll
      for (int i4 = (j + 1) / 4; i4 < DELTA_CHUNK / 4; i4++) {
        const float4 a = *reinterpret_cast<const float4*>(at + j * PREP_A_STRIDE + i4 * 4);
        if (i4 * 4 > j) x[i4 * 4] = fmaf(-a.x, x[j], x[i4 * 4]);
        if (i4 * 4 + 1 > j) x[i4 * 4 + 1] = fmaf(-a.y, x[j], x[i4 * 4 + 1]);
        if (i4 * 4 + 2 > j) x[i4 * 4 + 2] = fmaf(-a.z, x[j], x[i4 * 4 + 2]);
        x[i4 * 4 + 3] = fmaf(-a.w, x[j], x[i4 * 4 + 3]);
      }
    }
    float* dst = column < dp ? w + column : u + (column - dp);
    const int step = column < dp ? dp : p.v_pad;
#pragma unroll
    for (int i = 0; i < DELTA_CHUNK; i++) dst[(size_t)i * step] = x[i];
  }
}

// One block per (request, head, 16 value columns) walks the request's chunks with its columns of the state in shared memory.
template <typename T>
__global__ void __launch_bounds__(DELTA_THREADS)
delta_carry_kernel(const DeltaParams<T> p, int buffers) {
  extern __shared__ float4 carry_smem[];
  const int dim = p.dim, dp = p.dim_pad, ds = dp + 4, vp = p.v_pad, vdim = p.vdim;
  float* S = reinterpret_cast<float*>(carry_smem);        // [dp][20], 16 columns used
  float* us = S + dp * CARRY_STRIDE;                      // [64][16]
  float* part = us + DELTA_CHUNK * CARRY_COLS;            // [4][64][20], or the second half's sums [dp][20]
  const int part_floats = max(4 * DELTA_CHUNK, dp) * CARRY_STRIDE;
  float* tiles = part + part_floats;                      // per buffer W [64][ds], keys [64][dp]
  const int tile_floats = DELTA_CHUNK * (ds + dp);
  pdl_launch_dependents();
  pdl_wait();
  const int r = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * CARRY_COLS, tid = threadIdx.x;
  const int tokens = p.q_start[r + 1] - p.q_start[r], chunks = (tokens + DELTA_CHUNK - 1) / DELTA_CHUNK;
  if (chunks <= 0) return;
  const int slot = p.state_slots[r];
  if (slot < 0 || slot >= p.num_slots) {
    if (tid == 0) atomicOr(p.status, SPROUT_STATUS_BAD_PAGE);
    return;
  }
  int base = 0;
  for (int i = 0; i < r; i++) base += (p.q_start[i + 1] - p.q_start[i] + DELTA_CHUNK - 1) / DELTA_CHUNK;
  float* mine = p.state + (((size_t)slot * p.heads + h) * dim) * vdim;
  for (int e = tid; e < dp * CARRY_COLS; e += DELTA_THREADS) {
    const int d = e / CARRY_COLS, c = col0 + e % CARRY_COLS;
    S[d * CARRY_STRIDE + e % CARRY_COLS] = d < dim && c < vdim ? mine[(size_t)d * vdim + c] : 0.f;
  }
  auto load = [&](int c, int buf) {
    const size_t place = (size_t)(base + c) * p.heads + h;
    const float* w = p.w + place * DELTA_CHUNK * dp;
    const float* kd = p.kd + place * DELTA_CHUNK * dp;
    float* tw = tiles + buf * tile_floats;
    float* tk = tw + DELTA_CHUNK * ds;
    const int quads = dp / 4;
    for (int e = tid; e < DELTA_CHUNK * quads; e += DELTA_THREADS) {
      const int i = e / quads, d = (e % quads) * 4;
      dr_cp_async16(tw + i * ds + d, w + i * dp + d);
      dr_cp_async16(tk + i * dp + d, kd + i * dp + d);
    }
  };
  load(0, 0);
  dr_cp_commit();
  // the thread's part of U0 and the chunk's decay, fetched a chunk ahead
  const int ui = tid >> 2, uc = (tid & 3) * 4;
  const bool u_there = col0 + uc < vp;
  auto u_at = [&](int c) {
    return reinterpret_cast<float4*>(p.u + ((size_t)(base + c) * p.heads + h) * DELTA_CHUNK * vp + (size_t)ui * vp + col0 + uc);
  };
  float4 next_u = u_there ? *u_at(0) : make_float4(0.f, 0.f, 0.f, 0.f);
  float next_decay = p.decay[(size_t)base * p.heads + h];
  for (int c = 0; c < chunks; c++) {
    const int buf = buffers == 2 ? c & 1 : 0;
    float4 own = next_u;
    const float decay = next_decay;
    if (c + 1 < chunks) {
      if (u_there) next_u = *u_at(c + 1);
      next_decay = p.decay[(size_t)(base + c + 1) * p.heads + h];
    }
    if (buffers == 2 && c + 1 < chunks) {
      load(c + 1, buf ^ 1);
      dr_cp_commit();
      dr_cp_wait<1>();
    } else {
      dr_cp_wait<0>();
    }
    __syncthreads();                                      // the tiles have landed; S is whole
    const float* tw = tiles + buf * tile_floats;
    const float* tk = tw + DELTA_CHUNK * ds;
    const size_t place = (size_t)(base + c) * p.heads + h;
    {
      // W S: rows rt + 16 a, columns 4 ct .. 4 ct + 3, every fourth block of four d's
      const int rt = tid & 15, ct = (tid >> 4) & 3, ks = tid >> 6;
      float acc[4][4];
#pragma unroll
      for (int a = 0; a < 4; a++) acc[a][0] = acc[a][1] = acc[a][2] = acc[a][3] = 0.f;
      for (int d = ks * 4; d < dp; d += 16) {
        float4 s[4];
#pragma unroll
        for (int e = 0; e < 4; e++) s[e] = *reinterpret_cast<const float4*>(S + (d + e) * CARRY_STRIDE + ct * 4);
#pragma unroll
        for (int a = 0; a < 4; a++) {
          const float4 x = *reinterpret_cast<const float4*>(tw + (rt + 16 * a) * ds + d);
          acc[a][0] = fmaf(x.x, s[0].x, fmaf(x.y, s[1].x, fmaf(x.z, s[2].x, fmaf(x.w, s[3].x, acc[a][0]))));
          acc[a][1] = fmaf(x.x, s[0].y, fmaf(x.y, s[1].y, fmaf(x.z, s[2].y, fmaf(x.w, s[3].y, acc[a][1]))));
          acc[a][2] = fmaf(x.x, s[0].z, fmaf(x.y, s[1].z, fmaf(x.z, s[2].z, fmaf(x.w, s[3].z, acc[a][2]))));
          acc[a][3] = fmaf(x.x, s[0].w, fmaf(x.y, s[1].w, fmaf(x.z, s[2].w, fmaf(x.w, s[3].w, acc[a][3]))));
        }
      }
#pragma unroll
      for (int a = 0; a < 4; a++)
        *reinterpret_cast<float4*>(part + (ks * DELTA_CHUNK + rt + 16 * a) * CARRY_STRIDE + ct * 4) =
            make_float4(acc[a][0], acc[a][1], acc[a][2], acc[a][3]);
    }
    __syncthreads();
    {
      float4 sum = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int ks = 0; ks < 4; ks++) {
        const float4 x = *reinterpret_cast<const float4*>(part + (ks * DELTA_CHUNK + ui) * CARRY_STRIDE + uc);
        sum.x += x.x; sum.y += x.y; sum.z += x.z; sum.w += x.w;
      }
      own.x -= sum.x; own.y -= sum.y; own.z -= sum.z; own.w -= sum.w;
      if (u_there) *u_at(c) = own;
      *reinterpret_cast<float4*>(us + ui * CARRY_COLS + uc) = own;
    }
    __syncthreads();
    {
      // S <- decay S + K~^T U: tiles of 4 rows x 4 columns of S, the chunk's tokens in two halves
      float* before = p.before + place * dp * vp;
      const int half = tid >> 7;
      for (int tile0 = 0; tile0 < dp; tile0 += 128) {
        const int tile = tile0 + (tid & 127), ct = tile & 3, d0 = (tile >> 2) * 4;
        const bool there = tile < dp;
        float acc[4][4];
#pragma unroll
        for (int a = 0; a < 4; a++) acc[a][0] = acc[a][1] = acc[a][2] = acc[a][3] = 0.f;
        if (there) {
#pragma unroll 8
          for (int jj = 0; jj < DELTA_CHUNK / 2; jj++) {
            const int j = half * (DELTA_CHUNK / 2) + jj;
            const float4 k = *reinterpret_cast<const float4*>(tk + j * dp + d0);
            const float4 x = *reinterpret_cast<const float4*>(us + j * CARRY_COLS + ct * 4);
            acc[0][0] = fmaf(k.x, x.x, acc[0][0]); acc[0][1] = fmaf(k.x, x.y, acc[0][1]); acc[0][2] = fmaf(k.x, x.z, acc[0][2]); acc[0][3] = fmaf(k.x, x.w, acc[0][3]);
            acc[1][0] = fmaf(k.y, x.x, acc[1][0]); acc[1][1] = fmaf(k.y, x.y, acc[1][1]); acc[1][2] = fmaf(k.y, x.z, acc[1][2]); acc[1][3] = fmaf(k.y, x.w, acc[1][3]);
            acc[2][0] = fmaf(k.z, x.x, acc[2][0]); acc[2][1] = fmaf(k.z, x.y, acc[2][1]); acc[2][2] = fmaf(k.z, x.z, acc[2][2]); acc[2][3] = fmaf(k.z, x.w, acc[2][3]);
            acc[3][0] = fmaf(k.w, x.x, acc[3][0]); acc[3][1] = fmaf(k.w, x.y, acc[3][1]); acc[3][2] = fmaf(k.w, x.z, acc[3][2]); acc[3][3] = fmaf(k.w, x.w, acc[3][3]);
          }
          if (half == 1) {
#pragma unroll
            for (int a = 0; a < 4; a++)
              *reinterpret_cast<float4*>(part + (d0 + a) * CARRY_STRIDE + ct * 4) = make_float4(acc[a][0], acc[a][1], acc[a][2], acc[a][3]);
          }
        }
        __syncthreads();
        if (there && half == 0) {
#pragma unroll
          for (int a = 0; a < 4; a++) {
            float4* at = reinterpret_cast<float4*>(S + (d0 + a) * CARRY_STRIDE + ct * 4);
            const float4 s = *at, more = *reinterpret_cast<const float4*>(part + (d0 + a) * CARRY_STRIDE + ct * 4);
            if (col0 + ct * 4 < vp) *reinterpret_cast<float4*>(before + (size_t)(d0 + a) * vp + col0 + ct * 4) = s;
            *at = make_float4(fmaf(decay, s.x, acc[a][0] + more.x), fmaf(decay, s.y, acc[a][1] + more.y),
                              fmaf(decay, s.z, acc[a][2] + more.z), fmaf(decay, s.w, acc[a][3] + more.w));
          }
        }
      }
    }
    if (buffers != 2 && c + 1 < chunks) {
      __syncthreads();                                    // everyone is done with the one buffer
      load(c + 1, 0);
      dr_cp_commit();
    }
  }
  __syncthreads();
  for (int e = tid; e < dp * CARRY_COLS; e += DELTA_THREADS) {
    const int d = e / CARRY_COLS, c = col0 + e % CARRY_COLS;
    if (d < dim && c < vdim) mine[(size_t)d * vdim + c] = S[d * CARRY_STRIDE + e % CARRY_COLS];
  }
}

// o = Q~ S_0 + scores U for (chunk, head, 64 columns): thread (ti, tj) has rows ti + 16 a and columns 4 tj .. 4 tj + 3.
template <typename T>
__global__ void __launch_bounds__(DELTA_THREADS)
delta_outputs_kernel(const DeltaParams<T> p) {
  extern __shared__ float4 out_smem[];
  const int dp = p.dim_pad, ds = dp + 4, vp = p.v_pad, vdim = p.vdim;
  float* sq = reinterpret_cast<float*>(out_smem);         // [64][ds]
  float* ss = sq + DELTA_CHUNK * ds;                      // [dp][64]
  float* sp = ss + dp * OUT_COLS;                         // [64][68]
  float* su = sp + DELTA_CHUNK * PREP_A_STRIDE;           // [64][64]
  pdl_launch_dependents();
  pdl_wait();
  int r, c;
  if (!delta_find_chunk(p.q_start, p.requests, blockIdx.x, r, c)) return;
  const int h = blockIdx.y, col0 = blockIdx.z * OUT_COLS, tid = threadIdx.x;
  const int first = p.q_start[r] + c * DELTA_CHUNK, n = min(DELTA_CHUNK, p.q_start[r + 1] - first);
  const size_t place = (size_t)blockIdx.x * p.heads + h;
  const float* qd = p.qd + place * DELTA_CHUNK * dp;
  const float* before = p.before + place * dp * vp;
  const float* scores = p.scores + place * DELTA_CHUNK * DELTA_CHUNK;
  const float* u = p.u + place * DELTA_CHUNK * vp;
  const int quads = dp / 4;
  for (int e = tid; e < DELTA_CHUNK * quads; e += DELTA_THREADS) {
    const int i = e / quads, d = (e % quads) * 4;
    dr_cp_async16(sq + i * ds + d, qd + i * dp + d);
  }
  for (int e = tid; e < dp * (OUT_COLS / 4); e += DELTA_THREADS) {
    const int d = e / (OUT_COLS / 4), x = (e % (OUT_COLS / 4)) * 4;
    if (col0 + x < vp) dr_cp_async16(ss + d * OUT_COLS + x, before + (size_t)d * vp + col0 + x);
    else *reinterpret_cast<float4*>(ss + d * OUT_COLS + x) = make_float4(0.f, 0.f, 0.f, 0.f);
  }
  for (int e = tid; e < DELTA_CHUNK * (DELTA_CHUNK / 4); e += DELTA_THREADS) {
    const int i = e / (DELTA_CHUNK / 4), x = (e % (DELTA_CHUNK / 4)) * 4;
    dr_cp_async16(sp + i * PREP_A_STRIDE + x, scores + i * DELTA_CHUNK + x);
    if (col0 + x < vp) dr_cp_async16(su + i * OUT_COLS + x, u + (size_t)i * vp + col0 + x);
    else *reinterpret_cast<float4*>(su + i * OUT_COLS + x) = make_float4(0.f, 0.f, 0.f, 0.f);
  }
  dr_cp_commit();
  dr_cp_wait<0>();
  __syncthreads();
  const int ti = tid >> 4, tj = tid & 15;
  float acc[4][4];
#pragma unroll
  for (int a = 0; a < 4; a++) acc[a][0] = acc[a][1] = acc[a][2] = acc[a][3] = 0.f;
  auto add = [&](float (&row)[4], const float4& x, const float4 (&s)[4]) {
    row[0] = fmaf(x.x, s[0].x, fmaf(x.y, s[1].x, fmaf(x.z, s[2].x, fmaf(x.w, s[3].x, row[0]))));
    row[1] = fmaf(x.x, s[0].y, fmaf(x.y, s[1].y, fmaf(x.z, s[2].y, fmaf(x.w, s[3].y, row[1]))));
    row[2] = fmaf(x.x, s[0].z, fmaf(x.y, s[1].z, fmaf(x.z, s[2].z, fmaf(x.w, s[3].z, row[2]))));
    row[3] = fmaf(x.x, s[0].w, fmaf(x.y, s[1].w, fmaf(x.z, s[2].w, fmaf(x.w, s[3].w, row[3]))));
  };
#pragma unroll 2
  for (int d = 0; d < dp; d += 4) {
    float4 s[4];
#pragma unroll
    for (int e = 0; e < 4; e++) s[e] = *reinterpret_cast<const float4*>(ss + (d + e) * OUT_COLS + tj * 4);
#pragma unroll
    for (int a = 0; a < 4; a++) add(acc[a], *reinterpret_cast<const float4*>(sq + (ti + 16 * a) * ds + d), s);
  }
#pragma unroll
  for (int b = 0; b < 4; b++)                              // the scores are zero above the diagonal: rows before the block are left out
#pragma unroll
    for (int j = b * 16; j < b * 16 + 16; j += 4) {
      float4 s[4];
#pragma unroll
      for (int e = 0; e < 4; e++) s[e] = *reinterpret_cast<const float4*>(su + (j + e) * OUT_COLS + tj * 4);
#pragma unroll
      for (int a = b; a < 4; a++) add(acc[a], *reinterpret_cast<const float4*>(sp + (ti + 16 * a) * PREP_A_STRIDE + j), s);
    }
#pragma unroll
  for (int a = 0; a < 4; a++) {
    const int i = ti + 16 * a, col = col0 + tj * 4;
    if (i >= n || col >= vdim) continue;
    float* dst = p.out + (size_t)(first + i) * p.heads * vdim + (size_t)h * vdim + col;
    if ((vdim & 3) == 0) {
      *reinterpret_cast<float4*>(dst) = make_float4(acc[a][0], acc[a][1], acc[a][2], acc[a][3]);
    } else {
#pragma unroll
      for (int e = 0; e < 4; e++)
        if (col + e < vdim) dst[e] = acc[a][e];
    }
  }
}

constexpr int DELTA_MAX_SMEM = 227 * 1024 - 1024;

size_t prepare_bytes(int dp) { return (size_t)(2 * DELTA_CHUNK * (dp + 4) + DELTA_CHUNK * PREP_A_STRIDE) * sizeof(float); }
size_t carry_bytes(int dp, int buffers) {
  const int part = 4 * DELTA_CHUNK > dp ? 4 * DELTA_CHUNK : dp;
  return (size_t)((dp + part) * CARRY_STRIDE + DELTA_CHUNK * CARRY_COLS + buffers * DELTA_CHUNK * (2 * dp + 4)) * sizeof(float);
}
size_t outputs_bytes(int dp) {
  return (size_t)(DELTA_CHUNK * (dp + 4) + dp * OUT_COLS + DELTA_CHUNK * PREP_A_STRIDE + DELTA_CHUNK * OUT_COLS) * sizeof(float);
}

template <typename T>
int launch_delta(const DeltaParams<T>& p, int max_chunks, cudaStream_t stream) {
  if (max_chunks == 0) {
    int slices_log2 = 0;
    while ((WALK_ROWS << slices_log2) < p.dim) slices_log2++;
    SPROUT_REQUIRE(slices_log2 <= 5, "delta_rule: key vectors too long (%d)", p.dim);
    const int slices = 1 << slices_log2, cb = WALK_THREADS / slices * WALK_COLS;
    const size_t smem = (size_t)WALK_BATCH * ((size_t)WALK_ROWS * slices * sizeof(float2) + (size_t)cb * sizeof(float) + sizeof(float4) + sizeof(float));
    SPROUT_REQUIRE(smem <= 48 * 1024, "delta_rule: shared memory");
    sprout_launch(delta_walk_kernel<T>, dim3(p.requests, p.heads, (p.vdim + cb - 1) / cb), dim3(WALK_THREADS), smem, stream, p, slices_log2);
    return sprout_check_launch("delta_walk");
  }
  const int dp = p.dim_pad, buffers = carry_bytes(dp, 2) <= (size_t)DELTA_MAX_SMEM ? 2 : 1;
  SPROUT_REQUIRE(carry_bytes(dp, buffers) <= (size_t)DELTA_MAX_SMEM && outputs_bytes(dp) <= (size_t)DELTA_MAX_SMEM && prepare_bytes(dp) <= (size_t)DELTA_MAX_SMEM,
                 "delta_rule: key vectors too long for the chunked form (%d)", p.dim);
  static bool prepared = false;
  if (!prepared) {
    cudaFuncSetAttribute(delta_prepare_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, DELTA_MAX_SMEM);
    cudaFuncSetAttribute(delta_carry_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, DELTA_MAX_SMEM);
    cudaFuncSetAttribute(delta_outputs_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, DELTA_MAX_SMEM);
    prepared = true;
  }
  sprout_launch(delta_prepare_kernel<T>, dim3(max_chunks, p.heads), dim3(DELTA_THREADS), prepare_bytes(dp), stream, p);
  if (int rc = sprout_check_launch("delta_prepare")) return rc;
  sprout_launch(delta_carry_kernel<T>, dim3(p.requests, p.heads, (p.v_pad + CARRY_COLS - 1) / CARRY_COLS), dim3(DELTA_THREADS),
                carry_bytes(dp, buffers), stream, p, buffers);
  if (int rc = sprout_check_launch("delta_carry")) return rc;
  sprout_launch(delta_outputs_kernel<T>, dim3(max_chunks, p.heads, (p.v_pad + OUT_COLS - 1) / OUT_COLS), dim3(DELTA_THREADS),
                outputs_bytes(dp), stream, p);
  return sprout_check_launch("delta_outputs");
}

}  // namespace

// Floats of scratch that the chunked form needs for `max_chunks` chunks.
SPROUT_API long long sprout_delta_scratch_floats(int max_chunks, int heads, int dim, int vdim) {
  const long long dp = (dim + 3) / 4 * 4, vp = (vdim + 3) / 4 * 4;
  return (long long)max_chunks * heads * (DELTA_CHUNK * (3 * dp + vp + DELTA_CHUNK) + dp * vp + 4);
}

// `max_chunks` 0: token by token.  Otherwise at least the number of 64-token chunks of all requests, with `scratch` of
// sprout_delta_scratch_floats(max_chunks, ...) floats on a 16-byte boundary.
SPROUT_API int sprout_delta_rule(const void* q, const void* k, const void* v, int stride, const void* b, const void* a, int gate_stride,
                                 int dtype, const float* a_log, const float* dt_bias, int requests, int heads, int groups, int dim,
                                 int vdim, float q_scale, float unit_eps, const int* q_start, const int* state_slots, float* state,
                                 int num_slots, float* out, int max_chunks, float* scratch, int* status, cudaStream_t stream) {
  SPROUT_REQUIRE(q && k && v && b && a && a_log && dt_bias && q_start && state_slots && state && out && status, "delta_rule: null pointer");
  SPROUT_REQUIRE(requests > 0 && heads > 0 && groups > 0 && heads % groups == 0 && dim > 0 && vdim > 0 && num_slots > 0 && unit_eps > 0.f,
                 "delta_rule: bad sizes");
  SPROUT_REQUIRE(heads <= 65535 && max_chunks >= 0 && (max_chunks == 0 || (scratch && ((uintptr_t)scratch & 15) == 0)), "delta_rule: the chunked form needs its scratch");
  const int dp = (dim + 3) / 4 * 4, vp = (vdim + 3) / 4 * 4;
  float* at = scratch;
  auto take = [&](long long floats) {
    float* start = at;
    if (at) at += floats;
    return start;
  };
  const long long places = (long long)max_chunks * heads;
  float* w = take(places * DELTA_CHUNK * dp);
  float* kd = take(places * DELTA_CHUNK * dp);
  float* qd = take(places * DELTA_CHUNK * dp);
  float* u = take(places * DELTA_CHUNK * vp);
  float* scores = take(places * DELTA_CHUNK * DELTA_CHUNK);
  float* before = take(places * dp * vp);
  float* decay = take(places);
  if (dtype == SPROUT_F32) {
    DeltaParams<float> p{(const float*)q, (const float*)k, (const float*)v, stride, (const float*)b, (const float*)a, gate_stride, a_log,
                         dt_bias, heads, groups, dim, vdim, requests, q_scale, unit_eps, q_start, state_slots, state, num_slots, out,
                         status, dp, vp, w, kd, qd, u, scores, before, decay};
    return launch_delta(p, max_chunks, stream);
  }
  if (dtype == SPROUT_BF16) {
    DeltaParams<__nv_bfloat16> p{(const __nv_bfloat16*)q, (const __nv_bfloat16*)k, (const __nv_bfloat16*)v, stride,
                                 (const __nv_bfloat16*)b, (const __nv_bfloat16*)a, gate_stride, a_log, dt_bias, heads, groups, dim,
                                 vdim, requests, q_scale, unit_eps, q_start, state_slots, state, num_slots, out, status, dp, vp, w,
                                 kd, qd, u, scores, before, decay};
    return launch_delta(p, max_chunks, stream);
  }
  return sprout_fail("delta_rule: unknown dtype %d", dtype);
}
