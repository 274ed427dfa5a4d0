// Linear attention with one constant decay per head, in chunks on tensor cores: per head, over a request's tokens,
//
//   S_t = a S_{t-1} + k_t v_t^T,   o_t = S_t^T q_t        (S [D key channels x V value channels], float32)
//
// A request's new tokens of a step are cut into pieces of RC tokens.  With S_in the state at a piece's start and
// n its tokens (numbered from 0),
//
//   o_i   = a^(i+1) S_in^T q_i + sum_{j <= i} a^(i-j) (q_i . k_j) v_j
//   S_out = a^n S_in + sum_j a^(n-1-j) k_j v_j^T
//
//   retention_local    the sum in S_out, for all pieces side by side
//   retention_carry    S_in of every piece, from the request's slot on, and the state behind the last into the slot
//   retention_output   both terms of o, for all pieces side by side
//
// A step that brings one token a request takes one kernel from the projection to the gated output (retention_step):
// rotation, state, read-out, unit norm and gate, all in float32.
//
// The operands are float32.  A product on the tensor cores takes each as the sum of two bfloat16 values and forms
// the three partial products that count, hi hi + hi lo + lo hi, with float32 sums: a relative error of about 2^-16
// an operand, decays, scores and the state included.  A result does not depend on how a prompt was cut or on what
// else a step carries beyond such roundings.
//
// Piece p of row r has the number row_q_start[r] / RC + r + p: distinct for all pieces of a step, and below
// tokens / RC + rows, which is what the workspace holds.
#include "common.cuh"
#include "mma.cuh"

namespace zb {

constexpr int RC = 64;                  // tokens of a piece
constexpr int RV = 64;                  // value columns of a tile
constexpr int R_THREADS = 256;
constexpr int R_VST = RV + 8;           // a row of a value tile or a state tile in shared memory

struct RetentionArgs {
  const float* q; long long q_stride;   // [tokens, .]: head h at column h * D
  const float* k; long long k_stride;
  const float* v; long long v_stride;   // head h at column h * V
  const float* decay;                   // [H]
  float* ws;                            // [pieces][H][D][V]: the pieces' sums, then the states at their starts
  float* out;                           // [tokens, H * V]
  float* state; long long slot_stride;  // slot s at state + s * slot_stride: [H][D][V]
  const int* slots; const int* row_q_start; const int* row_q_len;
  int rows, H, D, V, num_slots, write_state;
  int qk_vectors, v_vectors, state_vectors;    // rows move as 16-byte pieces
  int tiles_per_cta;                    // retention_output: value tiles a CTA walks
  int* status;
};

__device__ __forceinline__ int first_piece(const RetentionArgs& a, int row) { return a.row_q_start[row] / RC + row; }

// The row that a piece belongs to (-1: none); all threads of the block take part.
__device__ __forceinline__ int row_of_piece(const RetentionArgs& a, int piece, int* found) {
  if (threadIdx.x == 0) *found = -1;
  __syncthreads();
  for (int r = threadIdx.x; r < a.rows; r += blockDim.x) {
    const int p = piece - first_piece(a, r);
    if (p >= 0 && p * RC < a.row_q_len[r]) *found = r;       // at most one row
  }
  __syncthreads();
  return *found;
}

// Two floats as bfloat16 pairs hi and lo with x = hi + lo up to 2^-17.
__device__ __forceinline__ void split2(float x, float y, unsigned& hi, unsigned& lo) {
  hi = pack_bf16(x, y);
  lo = pack_bf16(x - __uint_as_float(hi << 16), y - __uint_as_float(hi & 0xffff0000u));
}

// rows x cols float32 from global (rows `stride` apart, the first `valid_rows` x `valid_cols` of them), row i times
// scale(i), into two shared-memory tiles of bfloat16, zeros elsewhere.  `cols` is a multiple of 4.
template <typename F>
__device__ __forceinline__ void load_split(__nv_bfloat16* hi, __nv_bfloat16* lo, int smem_stride, const float* src, long long stride,
                                           int rows, int cols, int valid_rows, int valid_cols, bool vectors, F scale) {
  // Eight loads are on their way before the first of them is waited for.
  constexpr int AHEAD = 8;
  const int per_row = cols / 4, total = rows * per_row;
  for (int e0 = threadIdx.x; e0 < total; e0 += R_THREADS * AHEAD) {
    float4 x[AHEAD];
#pragma unroll
    for (int u = 0; u < AHEAD; ++u) {
      const int e = e0 + u * R_THREADS, i = e / per_row, c = (e - i * per_row) * 4;
      x[u] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
      if (i < valid_rows && c < valid_cols) {
        const float* p = src + i * stride + c;
        if (vectors) {                  // valid_cols is a multiple of 4 then
          x[u] = *reinterpret_cast<const float4*>(p);
        } else {
          x[u].x = p[0];
          if (c + 1 < valid_cols) x[u].y = p[1];
          if (c + 2 < valid_cols) x[u].z = p[2];
          if (c + 3 < valid_cols) x[u].w = p[3];
        }
      }
    }
#pragma unroll
    for (int u = 0; u < AHEAD; ++u) {
      const int e = e0 + u * R_THREADS, i = e / per_row, c = (e - i * per_row) * 4;
      if (e >= total) break;
      const float s = i < valid_rows ? scale(i) : 0.0f;
      uint2 h, l;
      split2(x[u].x * s, x[u].y * s, h.x, l.x);
      split2(x[u].z * s, x[u].w * s, h.y, l.y);
      *reinterpret_cast<uint2*>(hi + i * smem_stride + c) = h;
      *reinterpret_cast<uint2*>(lo + i * smem_stride + c) = l;
    }
  }
}

// acc (16 x 16 N) += A (16 x 16, hi and lo) * B (16 x 16 N), B stored [k][R_VST] in hi and lo tiles, from this lane's
// ldmatrix addresses inside the first 16 x 16 block on.
template <int N>
__device__ __forceinline__ void mma_rows_by_tile(float (&acc)[2 * N][4], const unsigned (&ah)[4], const unsigned (&al)[4],
                                                 const __nv_bfloat16* hi, const __nv_bfloat16* lo) {
#pragma unroll
  for (int n = 0; n < N; ++n) {
    unsigned bh[4], bl[4];
    ldmatrix_x4_trans(bh, hi + n * 16);
    ldmatrix_x4_trans(bl, lo + n * 16);
    mma_bf16_16816(acc[2 * n], al, bh[0], bh[1]);            // the small products first
    mma_bf16_16816(acc[2 * n + 1], al, bh[2], bh[3]);
    mma_bf16_16816(acc[2 * n], ah, bl[0], bl[1]);
    mma_bf16_16816(acc[2 * n + 1], ah, bl[2], bl[3]);
    mma_bf16_16816(acc[2 * n], ah, bh[0], bh[1]);
    mma_bf16_16816(acc[2 * n + 1], ah, bh[2], bh[3]);
  }
}

__host__ __device__ constexpr int retention_kst(int D) { return (D + 15) / 16 * 16 + 8; }

// ws[piece][h] = sum_j a^(n-1-j) k_j v_j^T, 64 value columns a CTA.
__global__ void __launch_bounds__(R_THREADS) retention_local_kernel(const RetentionArgs a) {
  extern __shared__ __align__(16) unsigned char r_smem[];
  __shared__ int found;
  __shared__ float power_s[RC];
  const int piece = blockIdx.z, h = blockIdx.y, v0 = blockIdx.x * RV;
  const int row = row_of_piece(a, piece, &found);
  if (row < 0) return;
  const int kst = retention_kst(a.D), dk = (a.D + 15) / 16;
  __nv_bfloat16* k_hi = reinterpret_cast<__nv_bfloat16*>(r_smem);
  __nv_bfloat16* k_lo = k_hi + RC * kst;
  __nv_bfloat16* v_hi = k_lo + RC * kst;
  __nv_bfloat16* v_lo = v_hi + RC * R_VST;
  const int begin = (piece - first_piece(a, row)) * RC, n = min(RC, a.row_q_len[row] - begin);
  const long long t0 = a.row_q_start[row] + begin;
  if (threadIdx.x < RC) power_s[threadIdx.x] = powf(a.decay[h], static_cast<float>(threadIdx.x));
  __syncthreads();
  load_split(k_hi, k_lo, kst, a.k + t0 * a.k_stride + h * a.D, a.k_stride, RC, dk * 16, n, a.D, a.qk_vectors,
             [&](int i) { return power_s[n - 1 - i]; });
  load_split(v_hi, v_lo, R_VST, a.v + t0 * a.v_stride + h * a.V + v0, a.v_stride, RC, RV, n, min(RV, a.V - v0), a.v_vectors,
             [](int) { return 1.0f; });
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int a_off = ((lane & 7) + (lane >> 4) * 8) * kst + ((lane >> 3) & 1) * 8;                  // tokens x channels, transposed
  const int b_off = ((lane & 7) + ((lane >> 3) & 1) * 8) * R_VST + (lane >> 4) * 8;
  const int steps = (n + 15) / 16;
  float* dst = a.ws + (static_cast<long long>(piece) * a.H + h) * a.D * a.V;
  for (int mt = warp; mt < dk; mt += R_THREADS / 32) {
    float acc[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.0f;
    for (int ks = 0; ks < steps; ++ks) {
      unsigned ah[4], al[4];
      ldmatrix_x4_trans(ah, k_hi + ks * 16 * kst + mt * 16 + a_off);
      ldmatrix_x4_trans(al, k_lo + ks * 16 * kst + mt * 16 + a_off);
      mma_rows_by_tile<4>(acc, ah, al, v_hi + ks * 16 * R_VST + b_off, v_lo + ks * 16 * R_VST + b_off);
    }
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int d = mt * 16 + g + 8 * half, c = v0 + i * 8 + 2 * t;
        if (d >= a.D || c >= a.V) continue;
        float* p = dst + static_cast<long long>(d) * a.V + c;
        if (a.V % 2 == 0) {
          *reinterpret_cast<float2*>(p) = make_float2(acc[i][2 * half], acc[i][2 * half + 1]);
        } else {
          p[0] = acc[i][2 * half];
          if (c + 1 < a.V) p[1] = acc[i][2 * half + 1];
        }
      }
  }
}

// ws[piece] <- the state at the piece's start; the slot <- the state behind the row's last piece.  A thread owns PER
// neighbouring elements of a row's state and walks its pieces.
template <int PER>
__global__ void __launch_bounds__(128) retention_carry_kernel(const RetentionArgs a) {
  const long long per = static_cast<long long>(a.H) * a.D * a.V;
  const long long e = (static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x) * PER;
  const int row = blockIdx.y;
  const int slot = a.slots[row];
  if (slot < 0 || slot >= a.num_slots) {
    if (blockIdx.x == 0 && threadIdx.x == 0) report(a.status, STATUS_ROW_OUT_OF_RANGE, slot, row);
    return;
  }
  if (e >= per) return;
  const int n = a.row_q_len[row], pieces = (n + RC - 1) / RC;
  const int h = static_cast<int>(e / (static_cast<long long>(a.D) * a.V));        // (PER divides D * V)
  const float decay = a.decay[h], whole = powf(decay, static_cast<float>(RC));
  const float rest = powf(decay, static_cast<float>(n - (pieces - 1) * RC));
  float* state = a.state + static_cast<long long>(slot) * a.slot_stride + e;
  float* ws = a.ws + first_piece(a, row) * per + e;
  auto load = [](float (&x)[PER], const float* p) {
    if (PER == 4) {
      const float4 v = *reinterpret_cast<const float4*>(p);
      x[0] = v.x; x[PER > 1 ? 1 : 0] = v.y; x[PER > 2 ? 2 : 0] = v.z; x[PER > 3 ? 3 : 0] = v.w;
    } else {
      x[0] = *p;
    }
  };
  auto store = [](float* p, const float (&x)[PER]) {
    if (PER == 4) *reinterpret_cast<float4*>(p) = make_float4(x[0], x[PER > 1 ? 1 : 0], x[PER > 2 ? 2 : 0], x[PER > 3 ? 3 : 0]);
    else *p = x[0];
  };
  float now[PER];
  load(now, state);
  constexpr int AHEAD = 8;
  for (int p0 = 0; p0 < pieces; p0 += AHEAD) {
    float sum[AHEAD][PER];
#pragma unroll
    for (int u = 0; u < AHEAD; ++u)
      if (p0 + u < pieces) load(sum[u], ws + (p0 + u) * per);
#pragma unroll
    for (int u = 0; u < AHEAD; ++u)
      if (p0 + u < pieces) {
        store(ws + (p0 + u) * per, now);
        const float factor = p0 + u + 1 < pieces ? whole : rest;
#pragma unroll
        for (int i = 0; i < PER; ++i) now[i] = fmaf(factor, now[i], sum[u][i]);
      }
  }
  if (a.write_state) store(state, now);
}

// The outputs of a piece's tokens for one head: the scores once, then value tile by value tile.  A warp owns 16 tokens
// and half the columns of a tile (two warps form the same scores).
__global__ void __launch_bounds__(R_THREADS, 2) retention_output_kernel(const RetentionArgs a) {
  extern __shared__ __align__(16) unsigned char r_smem[];
  __shared__ int found;
  __shared__ float power_s[RC + 1];
  const int piece = blockIdx.z, h = blockIdx.y;
  const int row = row_of_piece(a, piece, &found);
  if (row < 0) return;
  const int slot = a.slots[row];
  if (slot < 0 || slot >= a.num_slots) return;             // reported by the carry
  const int kst = retention_kst(a.D), dk = (a.D + 15) / 16;
  __nv_bfloat16* q_hi = reinterpret_cast<__nv_bfloat16*>(r_smem);
  __nv_bfloat16* q_lo = q_hi + RC * kst;
  __nv_bfloat16* k_hi = q_lo + RC * kst;
  __nv_bfloat16* k_lo = k_hi + RC * kst;
  // The value and state tiles lie where the keys were: nobody reads those once the scores are formed.
  __nv_bfloat16* v_hi = k_hi;
  __nv_bfloat16* v_lo = v_hi + RC * R_VST;
  __nv_bfloat16* s_hi = v_lo + RC * R_VST;
  __nv_bfloat16* s_lo = s_hi + dk * 16 * R_VST;
  const int begin = (piece - first_piece(a, row)) * RC, n = min(RC, a.row_q_len[row] - begin);
  const long long t0 = a.row_q_start[row] + begin;
  if (threadIdx.x <= RC) power_s[threadIdx.x] = powf(a.decay[h], static_cast<float>(threadIdx.x));
  auto one = [](int) { return 1.0f; };
  load_split(q_hi, q_lo, kst, a.q + t0 * a.q_stride + h * a.D, a.q_stride, RC, dk * 16, n, a.D, a.qk_vectors, one);
  load_split(k_hi, k_lo, kst, a.k + t0 * a.k_stride + h * a.D, a.k_stride, RC, dk * 16, n, a.D, a.qk_vectors, one);
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int wr = warp & 3, c_half = (warp >> 2) * (RV / 2);
  const int row0 = wr * 16;                                  // this warp's tokens of the piece
  const bool works = row0 < n;
  const int q_off = (row0 + (lane & 7) + ((lane >> 3) & 1) * 8) * kst + (lane >> 4) * 8;
  const int k_off = ((lane & 7) + (lane >> 4) * 8) * kst + ((lane >> 3) & 1) * 8;
  const int b_off = ((lane & 7) + ((lane >> 3) & 1) * 8) * R_VST + (lane >> 4) * 8 + c_half;
  // Scores of the keys up to this warp's last token, decayed, as the hi and lo parts of the next product's operand.
  unsigned ph[4][4], pl[4][4];
#pragma unroll
  for (int kg = 0; kg < 4; ++kg) {                           // 16 keys
    if (!works || kg > wr) continue;
    float s[2][4];
#pragma unroll
    for (int i = 0; i < 2; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.0f;
    for (int ks = 0; ks < dk; ++ks) {
      unsigned ah[4], al[4], bh[4], bl[4];
      ldmatrix_x4(ah, q_hi + q_off + ks * 16);
      ldmatrix_x4(al, q_lo + q_off + ks * 16);
      ldmatrix_x4(bh, k_hi + kg * 16 * kst + k_off + ks * 16);
      ldmatrix_x4(bl, k_lo + kg * 16 * kst + k_off + ks * 16);
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        mma_bf16_16816(s[i], al, bh[2 * i], bh[2 * i + 1]);
        mma_bf16_16816(s[i], ah, bl[2 * i], bl[2 * i + 1]);
        mma_bf16_16816(s[i], ah, bh[2 * i], bh[2 * i + 1]);
      }
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const int back = row0 + g + (c >= 2 ? 8 : 0) - (kg * 16 + i * 8 + 2 * t + (c & 1));
        s[i][c] = back >= 0 ? s[i][c] * power_s[back] : 0.0f;
      }
      split2(s[i][0], s[i][1], ph[kg][2 * i], pl[kg][2 * i]);
      split2(s[i][2], s[i][3], ph[kg][2 * i + 1], pl[kg][2 * i + 1]);
    }
  }
  const float lead0 = power_s[min(row0 + g + 1, RC)], lead1 = power_s[min(row0 + g + 9, RC)];
  const float* states = a.ws + (static_cast<long long>(piece) * a.H + h) * a.D * a.V;
  const int tiles = (a.V + RV - 1) / RV;
  const int tile_end = min(tiles, static_cast<int>(blockIdx.x + 1) * a.tiles_per_cta);
  for (int tile = blockIdx.x * a.tiles_per_cta; tile < tile_end; ++tile) {
    const int v0 = tile * RV, cols = min(RV, a.V - v0);
    __syncthreads();                                         // the keys, or the tile before, are read
    load_split(v_hi, v_lo, R_VST, a.v + t0 * a.v_stride + h * a.V + v0, a.v_stride, RC, RV, n, cols, a.v_vectors, one);
    load_split(s_hi, s_lo, R_VST, states + v0, a.V, dk * 16, RV, a.D, cols, a.state_vectors, one);
    __syncthreads();
    if (!works) continue;
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.0f;
    for (int ks = 0; ks < dk; ++ks) {
      unsigned ah[4], al[4];
      ldmatrix_x4(ah, q_hi + q_off + ks * 16);
      ldmatrix_x4(al, q_lo + q_off + ks * 16);
      mma_rows_by_tile<2>(acc, ah, al, s_hi + ks * 16 * R_VST + b_off, s_lo + ks * 16 * R_VST + b_off);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      acc[i][0] *= lead0; acc[i][1] *= lead0;
      acc[i][2] *= lead1; acc[i][3] *= lead1;
    }
#pragma unroll
    for (int kg = 0; kg < 4; ++kg)
      if (kg <= wr) mma_rows_by_tile<2>(acc, ph[kg], pl[kg], v_hi + kg * 16 * R_VST + b_off, v_lo + kg * 16 * R_VST + b_off);
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int token = row0 + g + 8 * half, c = v0 + c_half + i * 8 + 2 * t;
        if (token >= n || c >= a.V) continue;
        float* p = a.out + (t0 + token) * a.H * a.V + h * a.V + c;
        if (a.V % 2 == 0) {
          *reinterpret_cast<float2*>(p) = make_float2(acc[i][2 * half], acc[i][2 * half + 1]);
        } else {
          p[0] = acc[i][2 * half];
          if (c + 1 < a.V) p[1] = acc[i][2 * half + 1];
        }
      }
  }
}

// ------------------------------------------------------------------------------- one token a request
struct RetentionStepArgs {
  void* out;                            // [tokens, H * V]
  const float* projected;               // [tokens, stride]: q heads | k heads | v heads | gate
  long long stride;
  const float* freqs;                   // [rot_dims / 2]
  int rot_dims;
  float k_scale, eps;
  const float* decay;                   // [H]
  float* state; long long slot_stride;
  const int* slots; const int* row_q_start; const int* row_q_len; const int* positions;
  int H, D, V, num_slots, write_state;
  int* status;
};

constexpr int RS_THREADS = 256;

// A CTA owns a request and a head.  Its threads cut the state's D rows into groups of `RS_THREADS / columns` and walk
// them, PER neighbouring columns each; eight loads are on their way at a time.
template <typename T, int PER>
__global__ void __launch_bounds__(RS_THREADS) retention_step_kernel(const RetentionStepArgs a) {
  extern __shared__ float rs_smem[];
  __shared__ float scratch[33];
  float* q_s = rs_smem;                                    // [D]
  float* k_s = q_s + a.D;                                  // [D]
  float* o_s = k_s + a.D;                                  // [V]
  float* part_s = o_s + a.V;                               // [RS_THREADS * PER]
  const int h = blockIdx.x, row = blockIdx.y, tid = threadIdx.x;
  const int slot = a.slots[row], n = a.row_q_len[row];
  if (slot < 0 || slot >= a.num_slots || n != 1) {
    if (tid == 0) report(a.status, n != 1 ? STATUS_INTERNAL_CHECK : STATUS_ROW_OUT_OF_RANGE, n != 1 ? n : slot, row);
    return;
  }
  const long long t = a.row_q_start[row];
  const float* token = a.projected + t * a.stride;
  float* state = a.state + static_cast<long long>(slot) * a.slot_stride + static_cast<long long>(h) * a.D * a.V;
  // The head's state comes into the cache while queries and keys turn.
  for (long long line = tid; line * 32 < static_cast<long long>(a.D) * a.V; line += RS_THREADS)
    asm volatile("prefetch.global.L2 [%0];\n" ::"l"(state + line * 32));
  const float pos = static_cast<float>(a.positions[t]);
  const int half = a.rot_dims / 2, qk = a.H * a.D;
  for (int i = tid; i < a.D; i += RS_THREADS) {
    if (i >= half && i < a.rot_dims) continue;             // the partner of one below
    const float qu = token[h * a.D + i], ku = token[qk + h * a.D + i];
    if (i >= a.rot_dims) {
      q_s[i] = qu;
      k_s[i] = ku * a.k_scale;
      continue;
    }
    const float qv = token[h * a.D + i + half], kv = token[qk + h * a.D + i + half];
    float s, c;
    sincosf(pos * a.freqs[i], &s, &c);
    q_s[i] = qu * c - qv * s;
    q_s[i + half] = qv * c + qu * s;
    k_s[i] = (ku * c - kv * s) * a.k_scale;
    k_s[i + half] = (kv * c + ku * s) * a.k_scale;
  }
  __syncthreads();
  const float decay = a.decay[h];
  const float* values = token + 2 * qk + h * a.V;
  const int all = a.V / PER;                               // columns in runs of PER (PER divides V)
  float ss = 0.0f;
  for (int c0 = 0; c0 < all; c0 += RS_THREADS) {
    const int cols = min(RS_THREADS, all - c0), groups = RS_THREADS / cols;
    const int group = tid / cols, col = tid - group * cols, at = (c0 + col) * PER;
    float o[PER], v[PER];
#pragma unroll
    for (int u = 0; u < PER; ++u) {
      o[u] = 0.0f;
      v[u] = group < groups ? values[at + u] : 0.0f;
    }
    if (group < groups) {
      constexpr int AHEAD = 8;
      for (int d0 = group; d0 < a.D; d0 += groups * AHEAD) {
        float s[AHEAD][PER];
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) {
          const int d = d0 + i * groups;
          if (d < a.D) {
            const float* p = state + static_cast<long long>(d) * a.V + at;
            if (PER == 4) *reinterpret_cast<float4*>(&s[i][0]) = *reinterpret_cast<const float4*>(p);
            else s[i][0] = *p;
          }
        }
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) {
          const int d = d0 + i * groups;
          if (d < a.D) {
            const float kd = k_s[d], qd = q_s[d];
#pragma unroll
            for (int u = 0; u < PER; ++u) {
              s[i][u] = fmaf(decay, s[i][u], kd * v[u]);
              o[u] = fmaf(s[i][u], qd, o[u]);
            }
            if (a.write_state) {
              float* p = state + static_cast<long long>(d) * a.V + at;
              if (PER == 4) *reinterpret_cast<float4*>(p) = *reinterpret_cast<const float4*>(&s[i][0]);
              else *p = s[i][0];
            }
          }
        }
      }
#pragma unroll
      for (int u = 0; u < PER; ++u) part_s[(group * cols + col) * PER + u] = o[u];
    }
    __syncthreads();
    for (int c = tid; c < cols * PER; c += RS_THREADS) {
      float sum = 0.0f;
      for (int g = 0; g < groups; ++g) sum += part_s[g * cols * PER + c];
      o_s[c0 * PER + c] = sum;
      ss = fmaf(sum, sum, ss);
    }
    __syncthreads();
  }
  const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / static_cast<float>(a.V) + a.eps);
  const float* gate = token + 2 * qk + a.H * a.V + h * a.V;
  T* out = static_cast<T*>(a.out) + (t * a.H + h) * a.V;
  for (int c = tid; c < a.V; c += RS_THREADS) {
    const float g = gate[c];
    out[c] = from_float<T>(o_s[c] * inv * (g / (1.0f + expf(-g))));
  }
}

inline size_t retention_local_smem(int D) { return sizeof(__nv_bfloat16) * 2 * (static_cast<size_t>(RC) * retention_kst(D) + RC * R_VST); }
inline size_t retention_output_smem(int D) {
  const size_t keys = static_cast<size_t>(2) * RC * retention_kst(D);
  const size_t tiles = static_cast<size_t>(2) * (RC + (D + 15) / 16 * 16) * R_VST;
  return sizeof(__nv_bfloat16) * (keys + (keys > tiles ? keys : tiles));
}

}  // namespace zb

using namespace zb;

ZB_API int zb_retention_piece_tokens() { return RC; }
// The most key channels per head.
ZB_API int zb_retention_max_channels() { return 256; }

// ws: (tokens / piece tokens + rows) * H * D * V floats, contents irrelevant.  All operands float32; q, k, v with unit
// inner stride.  The rows' tokens lie behind one another in the stream, row_q_start ascending.
ZB_API int zb_retention(float* out, const float* q, long long q_stride, const float* k, long long k_stride, const float* v,
                        long long v_stride, const float* decay, float* state, long long slot_stride, const int* slots,
                        const int* row_q_start, const int* row_q_len, int rows, int tokens, int H, int D, int V, int num_slots,
                        int write_state, float* ws, int* status, void* stream) {
  if (rows < 0 || tokens < 0 || H <= 0 || D <= 0 || V <= 0 || num_slots <= 0 || (rows > 0 && ws == nullptr)) return ERR_BAD_ARGUMENT;
  if (D > zb_retention_max_channels() || H > 65535 || rows > 65535) return ERR_UNSUPPORTED;
  if (rows == 0 || tokens == 0) return OK;
  const int pieces = tokens / RC + rows;
  if (pieces > 65535) return ERR_UNSUPPORTED;
  auto aligned = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
  RetentionArgs a;
  a.q = q; a.q_stride = q_stride; a.k = k; a.k_stride = k_stride; a.v = v; a.v_stride = v_stride; a.decay = decay;
  a.ws = ws; a.out = out; a.state = state; a.slot_stride = slot_stride; a.slots = slots; a.row_q_start = row_q_start;
  a.row_q_len = row_q_len; a.rows = rows; a.H = H; a.D = D; a.V = V; a.num_slots = num_slots; a.write_state = write_state;
  a.status = status;
  a.qk_vectors = D % 4 == 0 && q_stride % 4 == 0 && k_stride % 4 == 0 && aligned(q) && aligned(k);
  a.v_vectors = V % 4 == 0 && v_stride % 4 == 0 && aligned(v);
  a.state_vectors = V % 4 == 0 && aligned(ws);
  const int tiles = (V + RV - 1) / RV;
  // A CTA walks a head's value tiles on one set of scores; few pieces are spread over more CTAs.
  a.tiles_per_cta = tiles;
  while (a.tiles_per_cta > 1 && static_cast<long long>(pieces) * H * ((tiles + a.tiles_per_cta - 1) / a.tiles_per_cta) < 296)
    a.tiles_per_cta = (a.tiles_per_cta + 1) / 2;
  auto s = static_cast<cudaStream_t>(stream);
  const size_t local_smem = retention_local_smem(D), output_smem = retention_output_smem(D);
  if (cuda_failed(cudaFuncSetAttribute(retention_local_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(local_smem))) ||
      cuda_failed(cudaFuncSetAttribute(retention_output_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(output_smem))))
    return ERR_CUDA;
  retention_local_kernel<<<dim3(tiles, H, pieces), R_THREADS, local_smem, s>>>(a);
  const long long per = static_cast<long long>(H) * D * V;
  const bool four = D * V % 4 == 0 && aligned(ws) && aligned(state) && slot_stride % 4 == 0;
  const long long threads = four ? per / 4 : per;
  const dim3 carry(static_cast<unsigned>((threads + 127) / 128), rows);
  if (four) retention_carry_kernel<4><<<carry, 128, 0, s>>>(a);
  else retention_carry_kernel<1><<<carry, 128, 0, s>>>(a);
  retention_output_kernel<<<dim3((tiles + a.tiles_per_cta - 1) / a.tiles_per_cta, H, pieces), R_THREADS, output_smem, s>>>(a);
  return launch_result();
}

// One token a request, from the projection's float32 rows (q | k | v | gate) to the gated, unit-normed output [tokens,
// H * V] in `dtype`, the requests' states brought up to date.
ZB_API int zb_retention_step(void* out, const float* projected, long long stride, const float* freqs, int rot_dims, float k_scale,
                             float eps, const float* decay, float* state, long long slot_stride, const int* slots,
                             const int* row_q_start, const int* row_q_len, const int* positions, int rows, int H, int D, int V,
                             int num_slots, int write_state, int dtype, int* status, void* stream) {
  if (rows < 0 || H <= 0 || D <= 0 || V <= 0 || num_slots <= 0 || rot_dims < 0 || rot_dims > D || rot_dims % 2 != 0 ||
      (rot_dims > 0 && freqs == nullptr) || stride < 2LL * H * (static_cast<long long>(D) + V))
    return ERR_BAD_ARGUMENT;
  if (rows > 65535 || 2LL * D + V > 10000) return ERR_UNSUPPORTED;
  if (rows == 0) return OK;
  RetentionStepArgs a;
  a.out = out; a.projected = projected; a.stride = stride; a.freqs = freqs; a.rot_dims = rot_dims; a.k_scale = k_scale; a.eps = eps;
  a.decay = decay; a.state = state; a.slot_stride = slot_stride; a.slots = slots; a.row_q_start = row_q_start;
  a.row_q_len = row_q_len; a.positions = positions; a.H = H; a.D = D; a.V = V; a.num_slots = num_slots;
  a.write_state = write_state; a.status = status;
  auto s = static_cast<cudaStream_t>(stream);
  const dim3 grid(H, rows);
  const bool four = V % 4 == 0 && slot_stride % 4 == 0 && reinterpret_cast<uintptr_t>(state) % 16 == 0;
  const size_t smem = sizeof(float) * (2 * D + V + RS_THREADS * (four ? 4 : 1));
  if (dtype == DTYPE_F32) {
    if (four) retention_step_kernel<float, 4><<<grid, RS_THREADS, smem, s>>>(a);
    else retention_step_kernel<float, 1><<<grid, RS_THREADS, smem, s>>>(a);
  } else {
    if (four) retention_step_kernel<__nv_bfloat16, 4><<<grid, RS_THREADS, smem, s>>>(a);
    else retention_step_kernel<__nv_bfloat16, 1><<<grid, RS_THREADS, smem, s>>>(a);
  }
  return launch_result();
}
