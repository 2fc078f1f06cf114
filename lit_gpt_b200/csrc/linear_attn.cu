// Decaying linear attention: a recurrent layer whose state is one dk x dv matrix S per head, kept in fp32.
//
//   per token:  S <- diag(g) S + k v^T      (g: one fixed decay per head, or one per head and key channel from the token)
//               o  = S^T q                  (the read-out sees the token's own write)
//   q, k, v come straight from the projections (bf16 or fp32), optionally through silu, q times a constant -- or q and k in fp32 from a
//   step of their own (a rotation) beside values in the projections' dtype; with per-channel
//   decays g = sigmoid(z + bias)^(1 / tau), all of it in fp32.
//
// walk_kernel goes through the tokens of one piece of a sequence in order.  The columns of S never mix: column j evolves from
// (k, q, g) and v[j] alone, so CTAs share out the columns, LK lanes of a warp hold the keys of NC neighbouring columns between them
// (KPL keys per lane, in registers, as pairs for the packed fp32 instructions), and a token costs each lane three packed operations
// per pair and column -- write, decay, read-out -- plus one short reduction over the LK lanes.  Tiles of tokens are staged in shared
// memory; the loads of the next tile are issued before the tokens of the current one are walked.
//
// Single tokens and short portions are one launch of it, from the slot's state to the slot's state.  Long prompts are cut into pieces
// that run side by side, because the recurrence is linear in the state:
//   1. walk every piece from S = 0 without read-out: its own contribution D and the product P of its decays;
//   2. scan_kernel: the state at the start of every piece, S <- P S + D from piece to piece, and the sequence's final state;
//   3. walk every piece from its starting state with read-out.
// No logarithm or quotient of decays is taken, so any decay in [0, 1] is safe.  A sequence that starts at position 0 starts from
// S = 0 whatever its slot holds.  The state is stored [head][dk][dv].
#include "common.cuh"

namespace b200 {

namespace {

constexpr int kLaThreads = 128, kLaTile = 1024, kLaNC = 4;   // kLaTile: floats of keys (queries, decays) staged per tile

struct LaArgs {
  const void* q; const void* k; const void* v;
  int64_t ldq, ldk, ldv;
  int act;
  float q_scale;
  const float* z; int64_t ldz;      // per-channel: raw decay projections (or, with z_ready, the decays themselves)
  const void* bias; float inv_tau;
  int z_ready;
  const float* head_decay;          // per head: fixed decays
  float* state; int64_t slot_stride;
  float* out; int64_t ldo;
  const int4* seqs;
  int heads, dk, dv;
  int piece, n_pieces;              // tokens per piece, pieces per sequence in the workspace
  float* ws_state;                  // [seq][piece][head][dk][dv]
  float* ws_prod;                   // [seq][piece][head][dk]
  int vec_k, vec_z, vec_v, vec_s;   // 16-byte accesses possible on q and k / z / v / the state
};

typedef unsigned long long f2;   // two packed floats
__device__ __forceinline__ f2 pk2(float a, float b) { f2 r; asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b)); return r; }
__device__ __forceinline__ void un2(f2 v, float& a, float& b) { asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v)); }
__device__ __forceinline__ f2 fma2(f2 a, f2 b, f2 c) { f2 r; asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c)); return r; }
__device__ __forceinline__ f2 mul2(f2 a, f2 b) { f2 r; asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b)); return r; }

// sigmoid(z)^(1 / tau) = exp(-softplus(-z) / tau), accurate at both ends
__device__ __forceinline__ float channel_decay(float z, float inv_tau) { return expf(-(fmaxf(-z, 0.f) + log1pf(expf(-fabsf(z)))) * inv_tau); }

template <typename T>
__device__ __forceinline__ float silu_f(float z) {
  if (sizeof(T) == 2) return __fdividef(z, 1.0f + __expf(-z));   // 16-bit projections: far below their own rounding
  return z / (1.0f + expf(-z));
}

// Eight neighbouring elements of a row as they lie in memory (zero beyond `n`): converted only when they are put into shared memory, so
// that nothing waits for the loads of the next tile while the current one is walked.
template <typename T>
struct alignas(16) Raw8 {
  T e[8];
  __device__ __forceinline__ void load(const T* row, int i0, int n, bool vec, bool ok) {
    uint4* w = reinterpret_cast<uint4*>(e);
    constexpr int W = sizeof(T) / 2;   // 16-byte words
#pragma unroll
    for (int j = 0; j < W; ++j) w[j] = make_uint4(0, 0, 0, 0);
    if (!ok) return;
    if (vec && i0 + 8 <= n) {
#pragma unroll
      for (int j = 0; j < W; ++j) w[j] = reinterpret_cast<const uint4*>(row + i0)[j];
    } else {
#pragma unroll
      for (int j = 0; j < 8; ++j) if (i0 + j < n) e[j] = row[i0 + j];
    }
  }
  __device__ __forceinline__ void floats(float (&f)[8]) const { load8(e, f); }
};

// MODE 0: slot state -> slot state with read-out; 1: from zero, contribution and decay product to the workspace, no read-out;
// 2: from the piece's starting state in the workspace, read-out only.
// T: dtype of the values (and of the per-channel decays' bias), TQ: of queries and keys.
template <typename T, typename TQ, int LK, int KPL, bool CHANNEL, int MODE>
__global__ void __launch_bounds__(kLaThreads, sizeof(TQ) == 2 && KPL <= 8 ? 5 : (sizeof(T) == 2 && KPL <= 8 ? 4 : 1)) walk_kernel(LaArgs A) {
  constexpr int NC = kLaNC, DKP = LK * KPL, TT = kLaTile / DKP, GROUPS = kLaThreads / LK, COLS = GROUPS * NC;
  constexpr int NVV = (TT * COLS / 8 + kLaThreads - 1) / kLaThreads;   // 8-column pieces of a value tile per thread
  constexpr int K4 = KPL / 4;
  extern __shared__ __align__(16) float la_smem[];
  float* const ks = la_smem;                                  // [TT][DKP]
  float* const qs = ks + kLaTile;                             // [TT][DKP]       (read-out only)
  float* const gs = qs + (MODE == 1 ? 0 : kLaTile);           // [TT][DKP]       (per-channel decay only)
  float* const vs = gs + (CHANNEL ? kLaTile : 0);             // [TT][COLS]
  griddep_launch();
  griddep_wait();
  const int tid = threadIdx.x, sub = tid % LK, grp = tid / LK;
  const int h = blockIdx.y;
  const int sidx = MODE == 0 ? (int)blockIdx.z : (int)blockIdx.z / A.n_pieces, piece = MODE == 0 ? 0 : (int)blockIdx.z % A.n_pieces;
  const int4 sq = A.seqs[sidx];
  const int begin = MODE == 0 ? 0 : piece * A.piece, end = MODE == 0 ? sq.y : min(sq.y, begin + A.piece);
  if (begin >= end) return;
  const int first = sq.x + begin, len = end - begin;
  const int dk = A.dk, dv = A.dv;
  const int col0 = (int)blockIdx.x * COLS, col = col0 + grp * NC;
  float* const slot = A.state + (int64_t)sq.w * A.slot_stride + (int64_t)h * dk * dv;
  const int64_t wrow = ((int64_t)sidx * A.n_pieces + piece) * A.heads + h;
  const float* const src = MODE == 0 ? slot : A.ws_state + wrow * dk * dv;
  float* const dst = MODE == 0 ? slot : A.ws_state + wrow * dk * dv;
  const bool vs4 = A.vec_s && col + NC <= dv;

  // this lane's keys: r4 * 4 LK + 4 sub + {0 .. 3}, r4 < KPL / 4
  f2 S[KPL / 2][NC];
#pragma unroll
  for (int r = 0; r < KPL / 2; ++r) {
    const int i = (r >> 1) * 4 * LK + 4 * sub + 2 * (r & 1);
    float a[2][NC];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
#pragma unroll
      for (int c = 0; c < NC; ++c) a[e][c] = 0.f;
      if (MODE != 1 && (MODE == 2 || sq.z > 0) && i + e < dk) {
        const float* p = src + (int64_t)(i + e) * dv + col;
        if (vs4) {
          const float4 t = *reinterpret_cast<const float4*>(p);
          a[e][0] = t.x; a[e][1] = t.y; a[e][2] = t.z; a[e][3] = t.w;
        } else {
#pragma unroll
          for (int c = 0; c < NC; ++c) if (col + c < dv) a[e][c] = p[c];
        }
      }
    }
#pragma unroll
    for (int c = 0; c < NC; ++c) S[r][c] = pk2(a[0][c], a[1][c]);
  }
  f2 P[MODE == 1 ? KPL / 2 : 1];
  if (MODE == 1) {
#pragma unroll
    for (int r = 0; r < KPL / 2; ++r) P[r] = pk2(1.f, 1.f);
  }
  const float hd = CHANNEL ? 0.f : A.head_decay[h];
  const f2 hd2 = pk2(hd, hd);

  const TQ* const kp = reinterpret_cast<const TQ*>(A.k) + (int64_t)h * dk;
  const TQ* const qp = reinterpret_cast<const TQ*>(A.q) + (int64_t)h * dk;
  const T* const vp = reinterpret_cast<const T*>(A.v) + (int64_t)h * dv;
  const int st = tid / (DKP / 8), si = (tid % (DKP / 8)) * 8;          // this thread's token of a tile and its eight keys there
  Raw8<TQ> rk, rq;
  Raw8<T> rv[NVV];
  Raw8<float> rz;
  auto load_tile = [&](int t0) {
    const int nt = min(TT, len - t0);
    const int64_t row = first + t0 + st;
    rk.load(kp + row * A.ldk, si, dk, A.vec_k, st < nt);
    if constexpr (MODE != 1) rq.load(qp + row * A.ldq, si, dk, A.vec_k, st < nt);
    if constexpr (CHANNEL) rz.load(A.z + row * A.ldz + (int64_t)h * dk, si, dk, A.vec_z, st < nt);
#pragma unroll
    for (int n = 0; n < NVV; ++n) {
      const int idx = tid + n * kLaThreads, t = idx / (COLS / 8), c = (idx % (COLS / 8)) * 8;
      rv[n].load(vp + (int64_t)(first + t0 + t) * A.ldv, col0 + c, dv, A.vec_v, t < nt && col0 + c < dv);
    }
  };
  auto store_tile = [&](int nt) {
    float f[8];
    auto activate = [&]() {
      if (A.act) {
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] = silu_f<T>(f[j]);
      }
    };
    if (st < nt) {
      rk.floats(f);
      activate();
      store8(ks + st * DKP + si, f);
      if constexpr (MODE != 1) {
        rq.floats(f);
        activate();
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] *= A.q_scale;
        store8(qs + st * DKP + si, f);
      }
      if constexpr (CHANNEL) {
        rz.floats(f);
        if (!A.z_ready) {
          const T* bias = reinterpret_cast<const T*>(A.bias) + (int64_t)h * dk;
#pragma unroll
          for (int j = 0; j < 8; ++j) f[j] = channel_decay(f[j] + (si + j < dk ? load_as_float(bias, si + j) : 0.f), A.inv_tau);
        }
        store8(gs + st * DKP + si, f);
      }
    }
#pragma unroll
    for (int n = 0; n < NVV; ++n) {
      const int idx = tid + n * kLaThreads, t = idx / (COLS / 8), c = (idx % (COLS / 8)) * 8;
      if (t < nt) {
        rv[n].floats(f);
        activate();
        store8(vs + t * COLS + c, f);
      }
    }
  };

  load_tile(0);
  for (int t0 = 0; t0 < len; t0 += TT) {
    const int nt = min(TT, len - t0);
    __syncthreads();                       // the previous tile's tokens are done with shared memory
    store_tile(nt);
    __syncthreads();
    if (t0 + TT < len) load_tile(t0 + TT);
    for (int t = 0; t < nt; ++t) {
      const float4 vv = *reinterpret_cast<const float4*>(vs + t * COLS + grp * NC);
      const f2 v2[NC] = {pk2(vv.x, vv.x), pk2(vv.y, vv.y), pk2(vv.z, vv.z), pk2(vv.w, vv.w)};
      f2 o[NC];
#pragma unroll
      for (int c = 0; c < NC; ++c) o[c] = 0ull;
#pragma unroll
      for (int r4 = 0; r4 < K4; ++r4) {
        const int at = t * DKP + r4 * 4 * LK + 4 * sub;
        const ulonglong2 k4 = *reinterpret_cast<const ulonglong2*>(ks + at);
        ulonglong2 q4 = make_ulonglong2(0, 0), g4 = make_ulonglong2(hd2, hd2);
        if constexpr (MODE != 1) q4 = *reinterpret_cast<const ulonglong2*>(qs + at);
        if constexpr (CHANNEL) g4 = *reinterpret_cast<const ulonglong2*>(gs + at);
#pragma unroll
        for (int p = 0; p < 2; ++p) {
          const f2 kk = p ? k4.y : k4.x, qq = p ? q4.y : q4.x, gg = p ? g4.y : g4.x;
          const int r = 2 * r4 + p;
          if (MODE == 1) P[r] = mul2(P[r], gg);
#pragma unroll
          for (int c = 0; c < NC; ++c) {
            S[r][c] = fma2(gg, S[r][c], mul2(kk, v2[c]));
            if (MODE != 1) o[c] = fma2(S[r][c], qq, o[c]);
          }
        }
      }
      if constexpr (MODE != 1) {
        // sum of four columns over LK lanes: the first two rounds also deal the columns out, so that lane group (sub / (LK / 4)) ends
        // with the total of its own column
        float a[NC];
#pragma unroll
        for (int c = 0; c < NC; ++c) { float lo, hi; un2(o[c], lo, hi); a[c] = lo + hi; }
        const bool h1 = sub & (LK / 2), h2 = sub & (LK / 4);
        float x0 = h1 ? a[2] : a[0], x1 = h1 ? a[3] : a[1];
        const float y0 = h1 ? a[0] : a[2], y1 = h1 ? a[1] : a[3];
        x0 += __shfl_xor_sync(0xffffffffu, y0, LK / 2);
        x1 += __shfl_xor_sync(0xffffffffu, y1, LK / 2);
        float z = h2 ? x1 : x0;
        z += __shfl_xor_sync(0xffffffffu, h2 ? x0 : x1, LK / 4);
#pragma unroll
        for (int d = LK / 8; d > 0; d >>= 1) z += __shfl_xor_sync(0xffffffffu, z, d);
        const int c = col + (h1 ? 2 : 0) + (h2 ? 1 : 0);
        if ((sub & (LK / 4 - 1)) == 0 && c < dv) A.out[(int64_t)(first + t0 + t) * A.ldo + (int64_t)h * dv + c] = z;
      }
    }
  }
  if constexpr (MODE != 2) {
#pragma unroll
    for (int r = 0; r < KPL / 2; ++r) {
      const int i = (r >> 1) * 4 * LK + 4 * sub + 2 * (r & 1);
      float a[2][NC];
#pragma unroll
      for (int c = 0; c < NC; ++c) un2(S[r][c], a[0][c], a[1][c]);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        if (i + e >= dk) continue;
        float* p = dst + (int64_t)(i + e) * dv + col;
        if (vs4) {
          *reinterpret_cast<float4*>(p) = make_float4(a[e][0], a[e][1], a[e][2], a[e][3]);
        } else {
#pragma unroll
          for (int c = 0; c < NC; ++c) if (col + c < dv) p[c] = a[e][c];
        }
      }
      if (MODE == 1 && blockIdx.x == 0 && grp == 0) {
        float p0, p1;
        un2(P[r], p0, p1);
        if (i < dk) A.ws_prod[wrow * dk + i] = p0;
        if (i + 1 < dk) A.ws_prod[wrow * dk + i + 1] = p1;
      }
    }
  }
}

// Starting states of a sequence's pieces: ws_state[piece] <- S, S <- P S + D, and the final S into the slot.  One thread per V
// neighbouring columns of a key; the pieces' contributions are fetched a few ahead of the recurrence.
template <int V>
__global__ void __launch_bounds__(256) scan_kernel(LaArgs A) {
  griddep_launch();
  griddep_wait();
  const int4 sq = A.seqs[blockIdx.z];
  const int n = (sq.y + A.piece - 1) / A.piece, h = blockIdx.y;
  const int64_t e = ((int64_t)blockIdx.x * 256 + threadIdx.x) * V, per = (int64_t)A.dk * A.dv;
  if (e >= per) return;
  const int i = (int)(e / A.dv);
  float* const slot = A.state + (int64_t)sq.w * A.slot_stride + h * per + e;
  const int64_t w0 = (int64_t)blockIdx.z * A.n_pieces * A.heads + h;
  float* const ws = A.ws_state + w0 * per + e;
  const float* const pr = A.ws_prod + w0 * A.dk + i;
  const int64_t wst = (int64_t)A.heads * per, pst = (int64_t)A.heads * A.dk;
  float S[V];
#pragma unroll
  for (int j = 0; j < V; ++j) S[j] = 0.f;
  auto ld = [&](const float* p, float (&f)[V]) {
    if constexpr (V == 4) { const float4 t = *reinterpret_cast<const float4*>(p); f[0] = t.x; f[1] = t.y; f[2] = t.z; f[3] = t.w; }
    else f[0] = *p;
  };
  auto stv = [&](float* p, const float (&f)[V]) {
    if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
    else *p = f[0];
  };
  if (sq.z > 0) ld(slot, S);
  constexpr int U = 8;
  for (int c0 = 0; c0 < n; c0 += U) {
    float D[U][V], P[U];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (c0 + u < n) { ld(ws + (c0 + u) * wst, D[u]); P[u] = pr[(c0 + u) * pst]; }
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (c0 + u >= n) continue;
      stv(ws + (c0 + u) * wst, S);
#pragma unroll
      for (int j = 0; j < V; ++j) S[j] = fmaf(P[u], S[j], D[u][j]);
    }
  }
  stv(slot, S);
}

// z <- sigmoid(z + bias)^(1 / tau) in place over rows of `cols` channels: a prompt's decays, once instead of once per column block
template <typename T>
__global__ void __launch_bounds__(256) decay_kernel(float* __restrict__ z, int64_t ldz, const T* __restrict__ bias, int64_t rows, int cols, float inv_tau) {
  griddep_launch();
  griddep_wait();
  const int64_t n = rows * cols;
  for (int64_t i = (int64_t)blockIdx.x * 256 + threadIdx.x; i < n; i += (int64_t)gridDim.x * 256) {
    const int64_t r = i / cols;
    const int c = (int)(i - r * cols);
    float* p = z + r * ldz + c;
    *p = channel_decay(*p + load_as_float(bias, c), inv_tau);
  }
}

template <typename T, typename TQ, int LK, int KPL, bool CHANNEL, int MODE>
cudaError_t walk_launch(const LaArgs& A, int n_seqs, cudaStream_t st) {
  constexpr int COLS = kLaThreads / LK * kLaNC, TT = kLaTile / (LK * KPL);
  const size_t smem = (size_t)((1 + (MODE != 1) + (CHANNEL ? 1 : 0)) * kLaTile + TT * COLS) * sizeof(float);
  const dim3 grid((unsigned)((A.dv + COLS - 1) / COLS), (unsigned)A.heads, (unsigned)(MODE == 0 ? n_seqs : n_seqs * A.n_pieces));
  return launch(walk_kernel<T, TQ, LK, KPL, CHANNEL, MODE>, grid, dim3(kLaThreads), smem, st, A);
}

template <typename T, typename TQ, int LK, int KPL, bool CHANNEL>
cudaError_t scan_launch(const LaArgs& A, int n_seqs, cudaStream_t st) {
  if (A.n_pieces <= 1) return walk_launch<T, TQ, LK, KPL, CHANNEL, 0>(A, n_seqs, st);
  cudaError_t e = walk_launch<T, TQ, LK, KPL, CHANNEL, 1>(A, n_seqs, st);
  if (e != cudaSuccess) return e;
  const bool v4 = A.vec_s && A.dv % 4 == 0;
  const int64_t per = (int64_t)A.dk * A.dv / (v4 ? 4 : 1);
  const dim3 grid((unsigned)((per + 255) / 256), (unsigned)A.heads, (unsigned)n_seqs);
  e = v4 ? launch(scan_kernel<4>, grid, dim3(256), 0, st, A) : launch(scan_kernel<1>, grid, dim3(256), 0, st, A);
  if (e != cudaSuccess) return e;
  return walk_launch<T, TQ, LK, KPL, CHANNEL, 2>(A, n_seqs, st);
}

// qk_f32: queries and keys are fp32 whatever T is (with fixed decays)
template <typename T, int LK, int KPL>
cudaError_t pick_launch(const LaArgs& A, int n_seqs, bool channel, bool qk_f32, cudaStream_t st) {
  if (channel) return scan_launch<T, T, LK, KPL, true>(A, n_seqs, st);
  if (qk_f32) return scan_launch<T, float, LK, KPL, false>(A, n_seqs, st);
  return scan_launch<T, T, LK, KPL, false>(A, n_seqs, st);
}

int la_cols(int dk) { return kLaThreads / (dk <= 64 ? 8 : dk <= 128 ? 16 : 32) * kLaNC; }

int g_la_piece = 0;

// Tokens per piece: enough pieces for a few CTAs per SM, none shorter than 32 tokens
int la_piece(int64_t rows, int max_rows, int heads, int dk, int dv) {
  if (g_la_piece > 0) return g_la_piece;
  const int64_t blocks = (int64_t)((dv + la_cols(dk) - 1) / la_cols(dk)) * heads;
  const int64_t want = (rows * blocks + (int64_t)sm_count() * 12 - 1) / ((int64_t)sm_count() * 12);
  int64_t p = (want + 15) / 16 * 16;
  return (int)(p < 32 ? 32 : p);
}

}  // namespace

}  // namespace b200

using namespace b200;

extern "C" {

int b200_linear_attn_tune(int piece) {
  const int old = g_la_piece;
  g_la_piece = piece > 0 ? piece : 0;
  return old;
}

size_t b200_linear_attn_workspace_bytes(int64_t rows, int max_rows, int n_seqs, int heads, int dk, int dv) {
  const int p = la_piece(rows, max_rows, heads, dk, dv);
  const int64_t pieces = (max_rows + p - 1) / p;
  return pieces <= 1 ? 0 : (size_t)n_seqs * pieces * heads * dk * (dv + 1) * sizeof(float);
}

int b200_linear_attn(const b200_linear_attn_args* a, b200_stream_t stream) {
  B200_CHECK_ARG(a && a->q && a->k && a->v && a->state && a->out && a->seqs, "b200_linear_attn: null pointer");
  B200_CHECK_ARG(!a->decay_in != !a->head_decay && (!a->decay_in || (a->decay_bias && a->tau > 0.f)),
                 "b200_linear_attn: either per-channel decays (raw, with bias and tau) or one fixed decay per head");
  B200_CHECK_ARG(a->n_seqs > 0 && a->heads > 0 && a->heads <= 65535 && a->rows > 0 && a->max_rows > 0 && a->max_rows <= a->rows, "b200_linear_attn: bad batch");
  B200_CHECK_ARG(a->dk > 0 && a->dk <= 512 && a->dv > 0, "b200_linear_attn: key size must be 1 .. 512");
  B200_CHECK_ARG(a->state_slot_stride >= (int64_t)a->heads * a->dk * a->dv, "b200_linear_attn: the state slots are too small");
  B200_CHECK_ARG((reinterpret_cast<uintptr_t>(a->seqs) & 15) == 0, "b200_linear_attn: seqs must be 16-byte aligned");
  const int piece = la_piece(a->rows, a->max_rows, a->heads, a->dk, a->dv);
  const int n_pieces = (a->max_rows + piece - 1) / piece;
  B200_CHECK_ARG((int64_t)a->n_seqs * n_pieces <= 65535, "b200_linear_attn: too many pieces");
  const size_t need = b200_linear_attn_workspace_bytes(a->rows, a->max_rows, a->n_seqs, a->heads, a->dk, a->dv);
  B200_CHECK_ARG(need == 0 || (a->workspace && a->workspace_bytes >= need), "b200_linear_attn: workspace too small (%zu of %zu bytes)", a->workspace_bytes, need);
  B200_CHECK_ARG(!a->qk_f32 || a->head_decay, "b200_linear_attn: fp32 queries and keys go with fixed decays");
  const size_t esz = a->dtype == B200_F32 ? 4 : 2, qsz = a->qk_f32 ? 4 : esz;
  auto al = [](const void* p, int64_t bytes) { return ((reinterpret_cast<uintptr_t>(p) | (uintptr_t)bytes) & 15) == 0; };
  float* const ws = (float*)a->workspace;
  const int64_t states = (int64_t)a->n_seqs * n_pieces * a->heads * a->dk * a->dv;
  LaArgs A{a->q, a->k, a->v, a->ldq, a->ldk, a->ldv, a->act, a->q_scale, a->decay_in, a->ld_decay, a->decay_bias, a->decay_in ? 1.0f / a->tau : 0.f, 0,
           a->head_decay, a->state, a->state_slot_stride, a->out, a->ldo, reinterpret_cast<const int4*>(a->seqs), a->heads, a->dk, a->dv, piece, n_pieces,
           ws, ws ? ws + states : nullptr,
           al(a->q, a->ldq * qsz) && al(a->k, a->ldk * qsz) && a->dk % 8 == 0, a->decay_in && al(a->decay_in, a->ld_decay * 4) && a->dk % 8 == 0,
           al(a->v, a->ldv * esz) && a->dv % 8 == 0, al(a->state, a->state_slot_stride * 4) && al(ws, 0) && a->dv % 4 == 0};
  cudaStream_t st = (cudaStream_t)stream;
  const bool ch = a->decay_in != nullptr;
  B200_FLOAT_TYPES(a->dtype, T, {
    if (ch && n_pieces > 1) {
      int64_t blocks = (a->rows * a->heads * a->dk + 255) / 256;
      const int64_t cap = (int64_t)sm_count() * 16;
      if (blocks > cap) blocks = cap;
      B200_CUDA(launch(decay_kernel<T>, dim3((unsigned)blocks), dim3(256), 0, st, a->decay_in, a->ld_decay, (const T*)a->decay_bias, a->rows,
                       a->heads * a->dk, A.inv_tau));
      A.z_ready = 1;
    }
    const bool qf = a->qk_f32 != 0;
    if (a->dk <= 32) B200_CUDA((pick_launch<T, 8, 4>(A, a->n_seqs, ch, qf, st)));
    else if (a->dk <= 64) B200_CUDA((pick_launch<T, 8, 8>(A, a->n_seqs, ch, qf, st)));
    else if (a->dk <= 128) B200_CUDA((pick_launch<T, 16, 8>(A, a->n_seqs, ch, qf, st)));
    else if (a->dk <= 256) B200_CUDA((pick_launch<T, 32, 8>(A, a->n_seqs, ch, qf, st)));
    else B200_CUDA((pick_launch<T, 32, 16>(A, a->n_seqs, ch, qf, st)));
  });
  return B200_OK;
}

}  // extern "C"
