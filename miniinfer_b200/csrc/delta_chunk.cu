// The gated delta rule with one decay a head, a chunk of 64 tokens at a time, in float32.
//
// With g_t the decay of a token, G_t the sum of ln g over the chunk up to and with token t, S_0 the state a chunk starts
// from [dim, vdim], and rows k_t, q_t, v_t, the recurrence
//   S_t = g_t S_(t-1) + k_t u_t^T,   u_t = beta_t (v_t - g_t S_(t-1)^T k_t),   o_t = S_t^T q_t
// is, over a chunk,
//   (I + L) U = diag(beta) (V - diag(e^G) K S_0),   L[t, s] = beta_t e^(G_t - G_s) (k_t . k_s)  for s < t,
//   O = diag(e^G) Q S_0 + A U,                      A[t, s] = e^(G_t - G_s) (q_t . k_s)         for s <= t,
//   S_C = e^(G_C) S_0 + (diag(e^(G_C - G)) K)^T U.
// The triangular system does not need the state if its right side is kept in two parts, U = U0 - W S_0 with
// (I + L) U0 = diag(beta) V and (I + L) W = diag(beta e^G) K.  All exponents are of sums of logarithms that are not positive.
// Three kernels:
//   chunk_solve  a block per (chunk, head), all at once: k . k, q . k, the triangular system by forward substitution - a
//                thread per column of [V | K], its 64 unknowns in registers -; W (transposed), U0 and A (transposed) to scratch;
//   chunk_state  a block per (request, head, 16 value columns), the only one that walks the chunks in order: keeps S, leaves
//                every chunk's S_0, U = U0 - W S_0 (over U0) and the state behind the last chunk;
//   chunk_out    a block per (chunk, head, 128 value columns), all at once: O, written over the values.
// Chunks are counted over the items of at least min_tokens new tokens, in their order; a step whose chunks need more
// scratch than SLAB_UNITS (chunk, head) pairs is worked through in slabs, the state row carrying over.
#include "delta_chunk.cuh"

namespace mi {
namespace {

constexpr int C = DELTA_CHUNK_TOKENS;
constexpr int SLAB_UNITS = 2048;
constexpr int THREADS = 256;
constexpr int CB = 16;                 // value columns of a chunk_state block
constexpr int OB = 128;                // value columns of a chunk_out block
constexpr int KT = 32;                 // inner values of a tile of chunk_out

__host__ __device__ inline int pad(int x, int m) { return (x + m - 1) / m * m; }

struct Args : DeltaChunkArgs {
  int dp, vp;                          // dim padded to 32, vdim padded to 16
  float *wt, *u, *at, *s0, *eg;        // per (chunk, head): W^T [dp][C], U0 / U [C][vp], A^T [C][C], S_0 [dp][vp], e^G [C] and e^(G_C - G) [C]
  int c0, c1;                          // the slab's chunks
};

__host__ __device__ inline long long unit_floats(int dp, int vp) { return (long long)dp * C + (long long)C * vp + C * C + (long long)dp * vp + 2 * C; }

// The item that chunk number c (over the items that are long enough) belongs to and the chunk's place in it; item -1: none.
__device__ __forceinline__ void find_chunk(const Args& a, int c, int& item, int& place) {
  item = -1;
  for (int b = 0; b < a.items; ++b) {
    const int n = a.q_len[b];
    if (n < a.min_tokens) continue;
    const int nc = (n + C - 1) / C;
    if (c < nc) { item = b; place = c; return; }
    c -= nc;
  }
}

__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ void st4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void copy16(float* dst, const float* src, bool take) {
  const unsigned d = (unsigned)__cvta_generic_to_shared(dst);
  const int bytes = take ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void copies_begun() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void copies_done() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// -------------------------------------------------------------------------------------------------------------- solve

__host__ __device__ inline size_t solve_smem(int dp) { return (size_t)(2 * C * (dp + 4) + 2 * C * C + 4 * C) * sizeof(float); }

__global__ void __launch_bounds__(THREADS, 2)
chunk_solve_kernel(Args a) {
  extern __shared__ __align__(16) float sm[];
  const int ld = a.dp + 4;
  float* ks = sm;                      // [C][ld]
  float* qs = ks + C * ld;             // [C][ld]
  float* lt = qs + C * ld;             // L^T [s][t]
  float* at = lt + C * C;              // A^T [s][t]
  float* bt = at + C * C;              // [C] beta
  float* eg = bt + C;                  // [C] e^G
  double* G = reinterpret_cast<double*>(eg + C);      // [C] sums of logarithms: differences of large sums keep their digits
  __shared__ int found[2];
  const int tid = threadIdx.x, head = blockIdx.y;
  if (tid == 0) find_chunk(a, a.c0 + blockIdx.x, found[0], found[1]);
  mi::grid_dependency_sync();
  __syncthreads();
  const int item = found[0];
  if (item < 0) return;
  const int first = found[1] * C, n = min(C, a.q_len[item] - first), row0 = a.q_start[item] + first;
  const int kvh = head / (a.heads / a.kv_heads);
  const size_t unit = (size_t)blockIdx.x * a.heads + head;
  {
    const int per_row = a.dp / 4, rows = THREADS / per_row, t0 = tid / per_row, d = (tid - t0 * per_row) * 4;
    for (int t = t0; t < C && t0 < rows; t += rows) {
      const bool in = t < n && d < a.dim;
      const size_t from = in ? ((size_t)(row0 + t) * a.kv_heads + kvh) * a.dim + d : 0;
      copy16(ks + t * ld + d, a.kn + from, in);
      copy16(qs + t * ld + d, a.qn + from, in);
    }
  }
  copies_begun();
  if (tid < 32) {                      // two tokens a lane (tokens behind the last: no decay, nothing written)
    const int t0 = 2 * tid, t1 = t0 + 1;
    const double x0 = t0 < n ? (double)a.lg[(size_t)(row0 + t0) * a.heads + head] : 0.0;
    const double x1 = t1 < n ? (double)a.lg[(size_t)(row0 + t1) * a.heads + head] : 0.0;
    double sum = x0 + x1;
    for (int o = 1; o < 32; o <<= 1) {
      const double y = __shfl_up_sync(0xffffffffu, sum, o);
      if (tid >= o) sum += y;
    }
    const double before = __shfl_up_sync(0xffffffffu, sum, 1), last = __shfl_sync(0xffffffffu, sum, 31);
    const double g0 = (tid > 0 ? before : 0.0) + x0, g1 = sum;
    G[t0] = g0;
    G[t1] = g1;
    eg[t0] = expf((float)g0);
    eg[t1] = expf((float)g1);
    bt[t0] = t0 < n ? a.beta[(size_t)(row0 + t0) * a.heads + head] : 0.f;
    bt[t1] = t1 < n ? a.beta[(size_t)(row0 + t1) * a.heads + head] : 0.f;
    float* e = a.eg + unit * 2 * C;
    e[t0] = eg[t0];
    e[t1] = eg[t1];
    e[C + t0] = expf((float)(last - g0));
    e[C + t1] = expf((float)(last - g1));
  }
  copies_done<0>();
  __syncthreads();
  {      // k . k and q . k: thread (tx, ty) has rows t = tx + 16 i and columns s = ty + 16 j; tiles above the diagonal are left out
    const int tx = tid & 15, ty = tid >> 4;
    float kk[4][4], qk[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) kk[i][j] = qk[i][j] = 0.f;
    for (int d = 0; d < a.dp; d += 4) {
      float4 kc[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) kc[j] = ld4(ks + (ty + 16 * j) * ld + d);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float4 kr = ld4(ks + (tx + 16 * i) * ld + d), qr = ld4(qs + (tx + 16 * i) * ld + d);
#pragma unroll
        for (int j = 0; j <= i; ++j) {
          kk[i][j] = fmaf(kr.x, kc[j].x, kk[i][j]); kk[i][j] = fmaf(kr.y, kc[j].y, kk[i][j]);
          kk[i][j] = fmaf(kr.z, kc[j].z, kk[i][j]); kk[i][j] = fmaf(kr.w, kc[j].w, kk[i][j]);
          qk[i][j] = fmaf(qr.x, kc[j].x, qk[i][j]); qk[i][j] = fmaf(qr.y, kc[j].y, qk[i][j]);
          qk[i][j] = fmaf(qr.z, kc[j].z, qk[i][j]); qk[i][j] = fmaf(qr.w, kc[j].w, qk[i][j]);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int t = tx + 16 * i, s = ty + 16 * j;
        const float e = s <= t ? expf((float)(G[t] - G[s])) : 0.f;
        lt[s * C + t] = s < t ? bt[t] * e * kk[i][j] : 0.f;
        at[s * C + t] = e * qk[i][j];
      }
  }
  __syncthreads();
  for (int i = tid; i < C * C / 4; i += THREADS) st4(a.at + unit * C * C + 4 * i, ld4(at + 4 * i));
  // the triangular system, a thread a column of [beta e^G K | beta V]; an unknown that is final is taken off all later rows
  for (int col = tid; col < a.dp + a.vp; col += THREADS) {
    const bool key = col < a.dp;
    const int c = col - a.dp;
    float x[C];
    if (key) {
#pragma unroll
      for (int t = 0; t < C; ++t) x[t] = bt[t] * eg[t] * ks[t * ld + col];
    } else {
      const float* v = a.raw + (size_t)row0 * (a.heads * a.vdim) + head * a.vdim + c;
      const bool in = c < a.vdim;
#pragma unroll
      for (int t = 0; t < C; ++t) x[t] = (in && t < n) ? bt[t] * v[(size_t)t * (a.heads * a.vdim)] : 0.f;
    }
#pragma unroll
    for (int s = 0; s < C - 1; ++s) {
#pragma unroll
      for (int t4 = (s + 1) / 4 * 4; t4 < C; t4 += 4) {
        const float4 l = ld4(lt + s * C + t4);
        if (t4 > s) x[t4] = fmaf(-l.x, x[s], x[t4]);
        if (t4 + 1 > s) x[t4 + 1] = fmaf(-l.y, x[s], x[t4 + 1]);
        if (t4 + 2 > s) x[t4 + 2] = fmaf(-l.z, x[s], x[t4 + 2]);
        if (t4 + 3 > s) x[t4 + 3] = fmaf(-l.w, x[s], x[t4 + 3]);
      }
    }
    if (key) {
      float* w = a.wt + unit * a.dp * C + (size_t)col * C;
#pragma unroll
      for (int t = 0; t < C; t += 4) st4(w + t, make_float4(x[t], x[t + 1], x[t + 2], x[t + 3]));
    } else {
      float* u = a.u + unit * C * a.vp + c;
#pragma unroll
      for (int t = 0; t < C; ++t) u[(size_t)t * a.vp] = x[t];
    }
  }
}

// -------------------------------------------------------------------------------------------------------------- state

__host__ __device__ inline size_t state_smem(int dp) {
  return (size_t)(2 * (dp * C + C * dp + C * CB + 2 * C) + dp * CB + C * CB + 8 * C * CB) * sizeof(float);
}

__global__ void __launch_bounds__(THREADS, 1)
chunk_state_kernel(Args a) {
  extern __shared__ __align__(16) float sm[];
  const int dp = a.dp, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int head = blockIdx.x, v0 = blockIdx.y * CB, item = blockIdx.z;
  const int n_new = a.q_len[item], row0 = a.q_start[item], slot = a.seq_slot[item];
  if (n_new < a.min_tokens) return;
  int base = 0;                        // the number of this item's first chunk
  for (int b = 0; b < item; ++b)
    if (a.q_len[b] >= a.min_tokens) base += (a.q_len[b] + C - 1) / C;
  const int from = max(a.c0, base), to = min(a.c1, base + (n_new + C - 1) / C);
  if (from >= to) return;
  const int kvh = head / (a.heads / a.kv_heads);
  const int buf_floats = 2 * dp * C + C * CB + 2 * C;
  float* bufs = sm;                    // two of: W^T [dp][C], K [C][dp], U0 [C][CB], e^G and e^(G_C - G) [2 C]
  float* S = bufs + 2 * buf_floats;    // [dp][CB]
  float* us = S + dp * CB;             // [C][CB] e^(G_C - G) U
  float* part = us + C * CB;           // [8][C][CB], a token's row at place t ^ ((t >> 2) & 1)
  mi::grid_dependency_sync();
  // which of K's 16-byte pieces this thread copies: one of a row, of every `rows`-th row
  const int per_row = dp / 4, rows = THREADS / per_row, kt = tid / per_row, kd = (tid - kt * per_row) * 4;
  auto fetch = [&](int c, float* buf) {
    const size_t unit = (size_t)(c - a.c0) * a.heads + head;
    const int first = (c - base) * C, n = min(C, n_new - first);
    const float* w = a.wt + unit * dp * C;
    for (int i = tid; i < dp * C / 4; i += THREADS) copy16(buf + 4 * i, w + 4 * i, true);
    float* kb = buf + dp * C;
    if (kt < rows) {
      const size_t step = (size_t)a.kv_heads * a.dim;
      const float* k = a.kn + (size_t)(row0 + first) * step + (size_t)kvh * a.dim + kd;
#pragma unroll 8
      for (int t = kt; t < C; t += rows) {
        const bool in = t < n && kd < a.dim;
        copy16(kb + t * dp + kd, in ? k + t * step : a.kn, in);
      }
    }
    float* ub = kb + C * dp;
    copy16(ub + 4 * tid, a.u + unit * C * a.vp + (size_t)(tid / 4) * a.vp + v0 + (tid % 4) * 4, true);      // C * CB / 4 = THREADS
    if (tid < 2 * C / 4) copy16(ub + C * CB + 4 * tid, a.eg + unit * 2 * C + 4 * tid, true);
    copies_begun();
  };
  fetch(from, bufs);
  // this thread's part of S: four rows, two columns (the blocks of narrower keys leave threads without one)
  const int d0 = (tid >> 3) * 4, cc = (tid & 7) * 2;
  const bool holds = d0 < dp;
  float* st = a.state + (size_t)slot * a.state_stride + (size_t)head * a.dim * a.vdim;
  float Sr[4][2];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int c = v0 + cc + j;
      Sr[i][j] = (d0 + i < a.dim && c < a.vdim) ? st[(size_t)(d0 + i) * a.vdim + c] : 0.f;
      if (holds) S[(d0 + i) * CB + cc + j] = Sr[i][j];
    }
  for (int c = from; c < to; ++c) {
    float* cur = bufs + (size_t)((c - from) & 1) * buf_floats;
    const size_t unit = (size_t)(c - a.c0) * a.heads + head;
    if (c + 1 < to) {
      fetch(c + 1, bufs + (size_t)((c + 1 - from) & 1) * buf_floats);
      copies_done<1>();
    } else {
      copies_done<0>();
    }
    __syncthreads();
    const float *w = cur, *kb = cur + dp * C, *ub = kb + C * dp, *ec = ub + C * CB + C;
    if (holds) {
#pragma unroll
      for (int i = 0; i < 4; ++i)
        *reinterpret_cast<float2*>(a.s0 + unit * dp * a.vp + (size_t)(d0 + i) * a.vp + v0 + cc) = make_float2(Sr[i][0], Sr[i][1]);
    }
    {      // W S_0: a warp takes an eighth of the key channels; a lane eight tokens and four columns
      const int rg = lane >> 2, cg = (lane & 3) * 4;
      float acc[8][4];
#pragma unroll
      for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
      const int per = dp / 8;
#pragma unroll 4
      for (int k = warp * per; k < (warp + 1) * per; ++k) {
        const float4 w0 = ld4(w + k * C + rg * 4), w1 = ld4(w + k * C + 32 + rg * 4), s = ld4(S + k * CB + cg);
        const float wr[8] = {w0.x, w0.y, w0.z, w0.w, w1.x, w1.y, w1.z, w1.w};
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          acc[i][0] = fmaf(wr[i], s.x, acc[i][0]); acc[i][1] = fmaf(wr[i], s.y, acc[i][1]);
          acc[i][2] = fmaf(wr[i], s.z, acc[i][2]); acc[i][3] = fmaf(wr[i], s.w, acc[i][3]);
        }
      }
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int t = (i < 4 ? 0 : 28) + rg * 4 + i;
        st4(part + ((size_t)warp * C + (t ^ (rg & 1))) * CB + cg, make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]));
      }
    }
    __syncthreads();
    {      // U = U0 - W S_0: a thread four columns of a token
      const int t = tid >> 2, cg = (tid & 3) * 4;
      float4 x = ld4(ub + t * CB + cg);
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        const float4 y = ld4(part + ((size_t)k * C + (t ^ ((t >> 2) & 1))) * CB + cg);
        x.x -= y.x; x.y -= y.y; x.z -= y.z; x.w -= y.w;
      }
      st4(a.u + unit * C * a.vp + (size_t)t * a.vp + v0 + cg, x);
      const float e = ec[t];
      st4(us + t * CB + cg, make_float4(e * x.x, e * x.y, e * x.z, e * x.w));
    }
    __syncthreads();
    if (holds) {      // S = e^(G_C) S_0 + K^T (e^(G_C - G) U)
      const float all = ec[-1];      // e^G of the chunk's last place
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j) Sr[i][j] *= all;
#pragma unroll 8
      for (int t = 0; t < C; ++t) {
        const float4 k4 = ld4(kb + t * dp + d0);
        const float2 u2 = *reinterpret_cast<const float2*>(us + t * CB + cc);
        Sr[0][0] = fmaf(k4.x, u2.x, Sr[0][0]); Sr[0][1] = fmaf(k4.x, u2.y, Sr[0][1]);
        Sr[1][0] = fmaf(k4.y, u2.x, Sr[1][0]); Sr[1][1] = fmaf(k4.y, u2.y, Sr[1][1]);
        Sr[2][0] = fmaf(k4.z, u2.x, Sr[2][0]); Sr[2][1] = fmaf(k4.z, u2.y, Sr[2][1]);
        Sr[3][0] = fmaf(k4.w, u2.x, Sr[3][0]); Sr[3][1] = fmaf(k4.w, u2.y, Sr[3][1]);
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) *reinterpret_cast<float2*>(S + (d0 + i) * CB + cc) = make_float2(Sr[i][0], Sr[i][1]);
    }
    __syncthreads();      // everyone is done with this buffer before the fetch after next fills it
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int c = v0 + cc + j;
      if (d0 + i < a.dim && c < a.vdim) st[(size_t)(d0 + i) * a.vdim + c] = Sr[i][j];
    }
}

// -------------------------------------------------------------------------------------------------------------- out

constexpr int RS = C + 4;              // a row of the transposed tile of tokens

__global__ void __launch_bounds__(THREADS, 3)
chunk_out_kernel(Args a) {
  __shared__ __align__(16) float rs[KT * RS];      // [KT][tokens]
  __shared__ __align__(16) float cs[KT * OB];      // [KT][value columns]
  __shared__ int found[2];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, head = blockIdx.y, v0 = blockIdx.z * OB;
  if (tid == 0) find_chunk(a, a.c0 + blockIdx.x, found[0], found[1]);
  mi::grid_dependency_sync();
  __syncthreads();
  const int item = found[0];
  if (item < 0) return;
  const int first = found[1] * C, n = min(C, a.q_len[item] - first), row0 = a.q_start[item] + first;
  const int kvh = head / (a.heads / a.kv_heads);
  const size_t unit = (size_t)blockIdx.x * a.heads + head;
  float acc[8][4];
#pragma unroll
  for (int i = 0; i < 8; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  auto columns = [&](const float* src) {      // KT rows of vp values
    for (int i = tid; i < KT * OB / 4; i += THREADS) {
      const int k = i / (OB / 4), c = (i % (OB / 4)) * 4;
      const bool in = v0 + c < a.vp;
      copy16(cs + k * OB + c, src + (in ? (size_t)k * a.vp + v0 + c : 0), in);
    }
  };
  auto multiply = [&]() {      // a warp eight tokens, a lane four columns
#pragma unroll 4
    for (int k = 0; k < KT; ++k) {
      const float4 r0 = ld4(rs + k * RS + warp * 8), r1 = ld4(rs + k * RS + warp * 8 + 4), x = ld4(cs + k * OB + lane * 4);
      const float r[8] = {r0.x, r0.y, r0.z, r0.w, r1.x, r1.y, r1.z, r1.w};
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        acc[i][0] = fmaf(r[i], x.x, acc[i][0]); acc[i][1] = fmaf(r[i], x.y, acc[i][1]);
        acc[i][2] = fmaf(r[i], x.z, acc[i][2]); acc[i][3] = fmaf(r[i], x.w, acc[i][3]);
      }
    }
  };
  for (int d0 = 0; d0 < a.dp; d0 += KT) {      // diag(e^G) Q S_0
    columns(a.s0 + unit * a.dp * a.vp + (size_t)d0 * a.vp);
    copies_begun();
    for (int i = tid; i < C * KT / 4; i += THREADS) {
      const int t = i / (KT / 4), d = (i % (KT / 4)) * 4;
      float4 q = make_float4(0.f, 0.f, 0.f, 0.f);
      if (t < n && d0 + d < a.dim) {
        const float e = a.eg[unit * 2 * C + t];
        q = ld4(a.qn + ((size_t)(row0 + t) * a.kv_heads + kvh) * a.dim + d0 + d);
        q.x *= e; q.y *= e; q.z *= e; q.w *= e;
      }
      rs[(d + 0) * RS + t] = q.x; rs[(d + 1) * RS + t] = q.y; rs[(d + 2) * RS + t] = q.z; rs[(d + 3) * RS + t] = q.w;
    }
    copies_done<0>();
    __syncthreads();
    multiply();
    __syncthreads();
  }
  for (int s0 = 0; s0 < C && s0 < n; s0 += KT) {      // A U
    columns(a.u + unit * C * a.vp + (size_t)s0 * a.vp);
    for (int i = tid; i < KT * C / 4; i += THREADS) copy16(rs + (i / (C / 4)) * RS + (i % (C / 4)) * 4, a.at + unit * C * C + (size_t)s0 * C + 4 * i, true);
    copies_begun();
    copies_done<0>();
    __syncthreads();
    multiply();
    __syncthreads();
  }
  const int c = v0 + lane * 4;
  if (c < a.vdim) {
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int t = warp * 8 + i;
      if (t < n) st4(a.raw + (size_t)(row0 + t) * (a.heads * a.vdim) + head * a.vdim + c, make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]));
    }
  }
}

int most_chunks(int T, int items) { return T / C + items; }      // every item's last chunk may be a short one
int slab_chunks(int heads) { return SLAB_UNITS / heads > 1 ? SLAB_UNITS / heads : 1; }

}  // namespace

long long delta_chunk_scratch_floats(int T, int items, int heads, int dim, int vdim) {
  const long long chunks = most_chunks(T, items) < slab_chunks(heads) ? most_chunks(T, items) : slab_chunks(heads);
  return chunks * heads * unit_floats(pad(dim, 32), pad(vdim, CB));
}

int delta_chunk_slabs(int T, int items, int heads) { return (most_chunks(T, items) + slab_chunks(heads) - 1) / slab_chunks(heads); }

int delta_chunk_run(const DeltaChunkArgs& in, int T, float* scratch, cudaStream_t stream) {
  MI_REQUIRE(in.dim > 0 && in.dim <= DELTA_CHUNK_MAX_DIM && in.dim % 4 == 0 && in.vdim % 4 == 0 && in.min_tokens > 0,
             "delta_chunk: dim=%d (a multiple of 4 up to %d), vdim=%d (a multiple of 4)", in.dim, DELTA_CHUNK_MAX_DIM, in.vdim);
  MI_REQUIRE(((uintptr_t)scratch % 16) == 0 && ((uintptr_t)in.qn % 16) == 0 && ((uintptr_t)in.kn % 16) == 0 && ((uintptr_t)in.raw % 16) == 0,
             "delta_chunk: buffers must be 16-byte aligned");
  Args a;
  static_cast<DeltaChunkArgs&>(a) = in;
  a.dp = pad(in.dim, 32);
  a.vp = pad(in.vdim, CB);
  const int total = most_chunks(T, in.items), slab = total < slab_chunks(in.heads) ? total : slab_chunks(in.heads);
  const size_t units = (size_t)slab * in.heads;
  a.wt = scratch;
  a.u = a.wt + units * a.dp * C;
  a.at = a.u + units * C * a.vp;
  a.s0 = a.at + units * C * C;
  a.eg = a.s0 + units * a.dp * a.vp;
  static bool configured = false;
  if (!configured) {
    cudaError_t e1 = cudaFuncSetAttribute(chunk_solve_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)solve_smem(DELTA_CHUNK_MAX_DIM));
    cudaError_t e2 = cudaFuncSetAttribute(chunk_state_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)state_smem(DELTA_CHUNK_MAX_DIM));
    if (e1 != cudaSuccess || e2 != cudaSuccess) return mi_fail("delta_chunk: the shared memory was refused");
    configured = true;
  }
  for (int c0 = 0; c0 < total; c0 += slab) {
    a.c0 = c0;
    a.c1 = c0 + slab < total ? c0 + slab : total;
    mi::launch(chunk_solve_kernel, dim3(a.c1 - a.c0, in.heads), dim3(THREADS), solve_smem(a.dp), stream, a);
    mi::launch(chunk_state_kernel, dim3(in.heads, a.vp / CB, in.items), dim3(THREADS), state_smem(a.dp), stream, a);
    mi::launch(chunk_out_kernel, dim3(a.c1 - a.c0, in.heads, (a.vp + OB - 1) / OB), dim3(THREADS), 0, stream, a);
  }
  MI_LAUNCH_OK("delta_chunk");
  return 0;
}

}  // namespace mi
