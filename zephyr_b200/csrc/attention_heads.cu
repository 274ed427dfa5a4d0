// Paged causal attention with ALL heads of a tile of tokens in one CTA, bfloat16 on tensor cores, for layers
// whose heads depend on one another between the scores and the softmax, and for keys and values of any two
// widths:
//
//   s_h(i, j) = scale q_h(i) . k_c(h)(j)              c(h) = h / (heads / kv_heads)
//   s_h <- sum_g M[h, g] s_g                          `score_mix` [nh, nh], or nothing
//   s_h <- s_h - r1_h ln(1 + r2_h (i - j))            `bias_r1`, `bias_r2` [nh], or nothing
//   softmax over the keys in sight (a window that may keep the first `keep_first` tokens), exp(sink_h) joining its
//   denominator where there are `sinks` [nh] (a key of that score with a value of zero), then the values
//
// The scores are float32 from the product to the softmax, the mixing included.
//
// One CTA = 8 or 16 consecutive new tokens of one request (or ONE decoded token), eight or sixteen warps of one or
// two heads each.  The products put keys on the 16-row side of m16n8k16 and tokens on its 8-column side
// (S^T = K Q^T, O^T = V^T P^T), so a warp keeps its heads' queries and outputs in registers whatever the count
// of tokens.  A tile of 32 (or 16) keys, with the
// keys and values of every key/value head, goes through three phases:
//   scores    each warp forms its heads' raw scores and leaves them in shared memory, [head][token][key];
//   mixing    S' = M S over the heads, for 8 keys of a token at a time, on the tensor cores and exact to float32: a
//             raw score is the sum of three bfloat16 values (24 bits), a matrix entry of one (an entry that is a
//             bfloat16 value, as in a bfloat16 checkpoint) or of three, and the products that count are added up in
//             float32; the bias is taken off, the mask applied, and the scores go back in place;
//   values    each warp reads its heads' scores as the second product's operand: online softmax in float32 in
//             base 2, probabilities rounded to bfloat16.
// The next tile's keys are fetched (16-byte asynchronous copies, straight from the pages) while this tile is
// mixed and weighed, its values while the next scores are formed.
//
// A decoded token's keys may be cut into `splits` runs of tiles, one CTA each; a second small kernel merges
// their partial results in the order of the context.  Math and masking as in attention_simt.cu.
#include "common.cuh"
#include "mma.cuh"

namespace zb {

constexpr size_t AH_SMEM_LIMIT = 227 * 1024;

struct HeadsAttentionArgs {
  const __nv_bfloat16* q;        // [T, nh * kd]
  __nv_bfloat16* out;            // [T, nh * vd]
  const __nv_bfloat16* kv_cache; // [num_pages]{[nkv][page_size][kd], [nkv][page_size][vd]}
  const int* block_table;        // [R, max_blocks]
  const int* tile_row;           // [n_tiles]
  const int* tile_q0;            // [n_tiles]
  const int* row_q_start;        // [R]
  const int* row_q_len;          // [R]
  const int* row_ctx;            // [R]
  int max_blocks, page_size, page_shift, num_pages, num_rows;      // page_shift: -1 where page_size is no power of two
  int nh, nkv, kd, vd, window, keep_first;
  float scale_log2;              // scale * log2(e)
  const float* score_mix;        // null, or [nh, nh]
  const float* bias_r1;          // null, or [nh] each
  const float* bias_r2;
  const float* sinks;            // null, or [nh]
  int splits;                    // > 1: every tile is one token, and its keys' tiles are shared by this many CTAs
  float* part_o;                 // [n_tiles, splits, nh, vd]
  float* part_ml;                // [n_tiles, splits, nh, 2]
  int* status;
};

__host__ __device__ constexpr int ah_head_stride(int tokens, int keys) { return tokens * (keys + 8) + 4; }
__host__ __device__ constexpr int ah_padded(int dim) { return (dim + 15) / 16 * 16 + 8; }      // a row in shared memory

// ldmatrix at a shared-memory address: the kernel's offsets are then plain 32-bit additions.
__device__ __forceinline__ void ah_ldmatrix(unsigned (&r)[4], unsigned address) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(address) : "memory");
}
__device__ __forceinline__ void ah_ldmatrix_trans(unsigned (&r)[4], unsigned address) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(address) : "memory");
}
__device__ __forceinline__ float ah_exp2(float x) {      // the special-function unit's: relative error about 2^-22
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void ah_copy16(unsigned smem, const void* gmem, int bytes) {       // 0 bytes: zeros
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(smem), "l"(gmem), "r"(bytes) : "memory");
}

// A float as the sum of three bfloat16 values, two floats at a time (the first in the low halves).
__device__ __forceinline__ void ah_split(float x, float y, unsigned& hi, unsigned& mid, unsigned& lo) {
  hi = pack_bf16(x, y);
  x -= __uint_as_float(hi << 16);
  y -= __uint_as_float(hi & 0xffff0000u);
  mid = pack_bf16(x, y);
  lo = pack_bf16(x - __uint_as_float(mid << 16), y - __uint_as_float(mid & 0xffff0000u));
}

// W warps in CG column groups; a warp has HPW heads and NT columns of 8 tokens.  DM: keys and values of up to 16 DM
// values, BK keys a tile.
template <int W, int HPW, int NT, int CG, int DM, int BK>
__global__ void __launch_bounds__(W * 32, W == 8 ? 2 : 1) heads_attention_kernel(const HeadsAttentionArgs a) {
  constexpr int THREADS = W * 32, WH = W / CG, HM = WH * HPW < 16 ? 16 : WH * HPW, NTOK = 8 * NT * CG, SST = BK + 8, MT = BK / 16;
  constexpr int HST = ah_head_stride(NTOK, BK);                        // floats between two heads' scores
  constexpr int MST = HM + 8;
  extern __shared__ __align__(16) unsigned char smem_raw[];
  const int kst = ah_padded(a.kd), vst = ah_padded(a.vd);
  __nv_bfloat16* k_s = reinterpret_cast<__nv_bfloat16*>(smem_raw);                     // [nkv][BK][kst]
  __nv_bfloat16* v_s = k_s + a.nkv * BK * kst;                                         // [nkv][BK][vst]
  __nv_bfloat16* mix_s = v_s + a.nkv * BK * vst;                                       // [3][HM][MST], the matrix's three parts
  float* s_s = reinterpret_cast<float*>(mix_s + 3 * HM * MST);                         // [HM][HST]: [NTOK][SST] of each head, zeros past the last
  // A tile's keys: where their first key/value head's key row and value row begin in the cache (bytes, multiples of
  // 16, the row's chunk permutation in the low bits; or bytes of any value for rows stored as they are), or -1 for a
  // key that nobody sees.
  __shared__ longlong2 where_s[2][BK];

  // The host lists the tiles by the number of keys they see, fewest first: the longest work starts first.
  const int tile = gridDim.y - 1 - blockIdx.y, split = blockIdx.x;
  const int row = a.tile_row[tile], q0 = a.tile_q0[tile];
  if (row < 0 || row >= a.num_rows) {
    if (threadIdx.x == 0) report(a.status, STATUS_ROW_OUT_OF_RANGE, row, tile);
    return;
  }
  const int q_len = a.row_q_len[row], ctx = a.row_ctx[row], tok0 = a.row_q_start[row] + q0;
  const int n_tok = min(a.splits > 1 ? 1 : NTOK, q_len - q0);
  if (n_tok <= 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int quad_row = lane >> 2, quad = lane & 3;
  const int* table = a.block_table + static_cast<size_t>(row) * a.max_blocks;
  const int ks_n = (a.kd + 15) / 16, vm_n = (a.vd + 15) / 16;

  // Keys any query of this tile may see: the kept first tokens below every window, and [lo, hi).
  const int hi = ctx + q0 + n_tok;
  const int lo = a.window > 0 ? max(0, ctx + q0 - a.window + 1) : 0;
  const int kept = a.window > 0 ? min(a.keep_first, lo) : 0;
  const int first_tile = lo / BK * BK;
  const int kept_tiles = (kept + BK - 1) / BK;
  const int all_tiles = kept_tiles + (hi - first_tile + BK - 1) / BK;
  const int t_begin = static_cast<int>(static_cast<long long>(all_tiles) * split / a.splits);
  const int t_end = static_cast<int>(static_cast<long long>(all_tiles) * (split + 1) / a.splits);
  auto tile_start = [&](int t) { return t < kept_tiles ? t * BK : first_tile + (t - kept_tiles) * BK; };

  const long long page_elems = static_cast<long long>(a.nkv) * a.page_size * (a.kd + a.vd);
  const long long value_part = static_cast<long long>(a.nkv) * a.page_size * a.kd;
  auto plan = [&](int t, int buffer) {               // by the first BK threads
    if (threadIdx.x >= BK) return;
    const int pos = tile_start(t) + static_cast<int>(threadIdx.x);
    int page = 0;
    if (t < kept_tiles ? pos < kept : (pos >= lo && pos < hi)) {
      const int block = a.page_shift >= 0 ? pos >> a.page_shift : pos / a.page_size;
      page = block < a.max_blocks ? table[block] : -1;
      if (page <= 0 || page >= a.num_pages) {
        report(a.status, STATUS_PAGE_OUT_OF_RANGE, page, tok0);
        page = 0;
      }
    }
    longlong2 at = make_longlong2(-1, -1);
    if (page > 0) {
      const int in_page = a.page_shift >= 0 ? pos & (a.page_size - 1) : pos % a.page_size;
      at.x = (page * page_elems + static_cast<long long>(in_page) * a.kd) * 2;
      at.y = (page * page_elems + value_part + static_cast<long long>(in_page) * a.vd) * 2;
      if (a.kd % 8 == 0) at.x += kv_swizzle(pos, a.kd / 8);
      if (a.vd % 8 == 0) at.y += kv_swizzle(pos, a.vd / 8);
    }
    where_s[buffer][threadIdx.x] = at;
  };
  // The planned tile's rows of every key/value head; zeros for keys that nobody sees.
  auto load_rows = [&](__nv_bfloat16* dst, int stride, int dim, bool values, int buffer) {
    const char* cache = reinterpret_cast<const char*>(a.kv_cache);
    if (dim % 8 == 0) {
      // A row's 16-byte pieces lie side by side on 4, 8, 16 or 32 lanes; a thread walks its keys, and for each of
      // them the key/value heads, whose rows lie a page's rows apart.
      const int chunks = dim / 8;
      const int shift = chunks <= 4 ? 2 : (chunks <= 8 ? 3 : (chunks <= 16 ? 4 : 5)), c = lane & ((1 << shift) - 1);
      if (c < chunks) {
        const unsigned step = static_cast<unsigned>(BK * stride) * 2u;
        const long long head_step = static_cast<long long>(a.page_size) * dim * 2;
        for (int key = (warp << (5 - shift)) + (lane >> shift); key < BK; key += W << (5 - shift)) {
          const long long from = values ? where_s[buffer][key].y : where_s[buffer][key].x;
          const bool seen = from >= 0;
          const char* src = cache + (seen ? (from & ~15LL) + ((c ^ static_cast<int>(from & 15)) << 4) : 0);
          const int bytes = seen ? 16 : 0;
          const long long advance = seen ? head_step : 0;
          unsigned to = smem_u32(dst + key * stride + c * 8);
#pragma unroll 4
          for (int kvh = 0; kvh < a.nkv; ++kvh, src += advance, to += step) ah_copy16(to, src, bytes);
        }
      }
    } else {                                           // rows stored as they are, on any boundary
      for (int r = warp; r < a.nkv * BK; r += W) {
        const int kvh = r / BK, key = r % BK;
        const long long from = values ? where_s[buffer][key].y : where_s[buffer][key].x;
        const __nv_bfloat16* src = reinterpret_cast<const __nv_bfloat16*>(
            cache + (from >= 0 ? from + static_cast<long long>(kvh) * a.page_size * dim * 2 : 0));
        for (int i = lane; i < dim; i += 32) dst[r * stride + i] = from >= 0 ? src[i] : __float2bfloat16_rn(0.0f);
      }
    }
  };
  auto load_keys = [&](int buffer) { load_rows(k_s, kst, a.kd, false, buffer); };
  auto load_values = [&](int buffer) { load_rows(v_s, vst, a.vd, true, buffer); };

  if (t_begin < t_end) plan(t_begin, 0);
  // The columns that pad a row to whole steps of 16 stay zero for good.
  for (int e = threadIdx.x; e < a.nkv * BK * (kst + vst) / 8; e += THREADS)
    reinterpret_cast<uint4*>(k_s)[e] = make_uint4(0, 0, 0, 0);
  for (int e = a.nh * HST + threadIdx.x; e < HM * HST; e += THREADS) s_s[e] = 0.0f;
  int inexact = 0;
  if (a.score_mix != nullptr)
    for (int e = threadIdx.x; e < HM * HM; e += THREADS) {
      const int h = e / HM, o = e - h * HM;
      float v = h < a.nh && o < a.nh ? a.score_mix[h * a.nh + o] : 0.0f;
#pragma unroll
      for (int part = 0; part < 3; ++part) {
        const __nv_bfloat16 b = __float2bfloat16_rn(v);
        mix_s[(part * HM + h) * MST + o] = b;
        v -= __bfloat162float(b);
        if (part == 0 && v != 0.0f) inexact = 1;
      }
    }
  const bool one_part = __syncthreads_or(inexact) == 0;      // (a barrier: the plan is there, the pads are zero)
  if (t_begin < t_end) load_keys(0);
  cp_async_commit();
  if (t_begin < t_end) load_values(0);
  cp_async_commit();

  // This warp's heads; their queries as the B operand (k = dims, n = tokens).  A head past the last one runs on the
  // last head's keys with queries of zero and is never stored.
  const int head0 = warp % WH * HPW, col0 = warp / WH * (8 * NT), g = a.nh / a.nkv;
  const bool works = head0 < a.nh && col0 < n_tok;
  unsigned k_at[HPW], v_at[HPW];                     // where this lane's rows of the heads' keys and values begin
  unsigned qf[HPW][NT][DM][2];
#pragma unroll
  for (int i = 0; i < HPW; ++i) {
    const int kvh = min(head0 + i, a.nh - 1) / g;
    k_at[i] = smem_u32(k_s + (kvh * BK + ((lane >> 3) & 1) * 8 + (lane & 7)) * kst + (lane >> 4) * 8);
    v_at[i] = smem_u32(v_s + (kvh * BK + (lane >> 4) * 8 + (lane & 7)) * vst + ((lane >> 3) & 1) * 8);
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) {
      const int tok = col0 + nt * 8 + quad_row, head = head0 + i;
      const bool ok = tok < n_tok && head < a.nh;
      const __nv_bfloat16* src = a.q + (static_cast<size_t>(tok0 + (ok ? tok : 0)) * a.nh + (ok ? head : 0)) * a.kd;
      const bool pairs = a.kd % 2 == 0;
#pragma unroll
      for (int ks = 0; ks < DM; ++ks) {
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int d = ks * 16 + half * 8 + 2 * quad;
          unsigned word = 0;
          if (ok && d < a.kd) {
            if (pairs) {
              word = *reinterpret_cast<const unsigned*>(src + d);
            } else {
              const __nv_bfloat162 two(src[d], d + 1 < a.kd ? src[d + 1] : __float2bfloat16_rn(0.0f));
              word = *reinterpret_cast<const unsigned*>(&two);
            }
          }
          qf[i][nt][ks][half] = word;
        }
      }
    }
  }
  float m_run[HPW][NT], l_run[HPW][NT];              // of token quad_row of each column
  float o[HPW][NT][DM][4];
#pragma unroll
  for (int i = 0; i < HPW; ++i)
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) {
      // A sink is a key that every token sees first, in the first split.
      const bool sink = a.sinks != nullptr && split == 0 && head0 + i < a.nh;
      m_run[i][nt] = sink ? a.sinks[head0 + i] * 1.4426950408889634f : -INFINITY;
      l_run[i][nt] = sink ? 1.0f : 0.0f;
#pragma unroll
      for (int m = 0; m < DM; ++m) o[i][nt][m][0] = o[i][nt][m][1] = o[i][nt][m][2] = o[i][nt][m][3] = 0.0f;
    }
  const unsigned k_step = static_cast<unsigned>(16 * kst) * 2u, v_step = static_cast<unsigned>(16 * vst) * 2u;   // 16 keys
  // In a piece of 8 keys: a lane's raw scores of two heads and one key, its final ones of one head and two keys, and its
  // rows of the mixing matrix.
  const int lane_raw = 2 * quad * HST + quad_row, lane_final = quad_row * HST + 2 * quad;
  const unsigned mix_at = smem_u32(mix_s + ((lane & 7) + ((lane >> 3) & 1) * 8) * MST + (lane >> 4) * 8);
  float* const raw_at = s_s + head0 * HST + (col0 + 2 * quad) * SST + quad_row;           // where this lane's raw scores go
  const float* const own_at = s_s + head0 * HST + (col0 + quad_row) * SST + 2 * quad;      // and where it reads its final ones

  cp_async_wait<1>();
  __syncthreads();                                   // the first tile's keys have landed
  for (int t = t_begin; t < t_end; ++t) {
    const int buffer = (t - t_begin) & 1;
    const bool more = t + 1 < t_end;
    if (more) plan(t + 1, buffer ^ 1);
    // ------------------------------------------------------------------------------------ raw scores
    if (works) {
      float acc[MT][HPW][NT][4];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int i = 0; i < HPW; ++i)
#pragma unroll
          for (int nt = 0; nt < NT; ++nt) acc[mt][i][nt][0] = acc[mt][i][nt][1] = acc[mt][i][nt][2] = acc[mt][i][nt][3] = 0.0f;
#pragma unroll
      for (int ks = 0; ks < DM; ++ks) {
        if (ks < ks_n) {
#pragma unroll
          for (int i = 0; i < HPW; ++i) {
#pragma unroll
            for (int mt = 0; mt < MT; ++mt) {
              unsigned ka[4];
              ah_ldmatrix(ka, k_at[i] + mt * k_step + ks * 32);
#pragma unroll
              for (int nt = 0; nt < NT; ++nt) mma_bf16_16816(acc[mt][i][nt], ka, qf[i][nt][ks][0], qf[i][nt][ks][1]);
            }
          }
        }
      }
#pragma unroll
      for (int i = 0; i < HPW; ++i) {
        if (head0 + i < a.nh) {
#pragma unroll
          for (int mt = 0; mt < MT; ++mt) {
#pragma unroll
            for (int nt = 0; nt < NT; ++nt) {
              float* dst = raw_at + i * HST + nt * 8 * SST + mt * 16;
              dst[0] = acc[mt][i][nt][0];
              dst[SST] = acc[mt][i][nt][1];
              dst[8] = acc[mt][i][nt][2];
              dst[SST + 8] = acc[mt][i][nt][3];
            }
          }
        }
      }
    }
    __syncthreads();                                 // every head's raw scores are there, the keys are read
    if (more) load_keys(buffer ^ 1);
    cp_async_commit();
    // --------------------------------------------------------------------- mixing, bias, mask, in place
    // A warp takes 8 keys of a token at a time, the same keys of every token it takes: the lane's columns are keys
    // 2 quad and 2 quad + 1, its rows heads.
    {
      constexpr int PER_TOKEN = BK / 8, TOKENS = W / PER_TOKEN, PIECES = (NTOK + TOKENS - 1) / TOKENS, AT_ONCE = HM == 16 ? 2 : 1;
      const int key8 = warp % PER_TOKEN * 8, tok_first = warp / PER_TOKEN;
      const int k0 = tile_start(t), pos = k0 + key8 + 2 * quad;
      // A tile that every token sees whole needs no mask: most tiles of a long window are such.
      const bool whole = t < kept_tiles ? k0 + BK <= kept
                                        : k0 + BK - 1 <= ctx + q0 && k0 >= lo && (a.window == 0 || k0 > hi - 1 - a.window);
      auto finish = [&](float* at, int tok, int h, float x, float y) {
        const int qp = ctx + q0 + tok;
        x *= a.scale_log2;
        y *= a.scale_log2;
        if (a.bias_r1 != nullptr) {
          const float r1 = a.bias_r1[h], r2 = a.bias_r2[h];
          x = fmaf(-r1, __log2f(fmaf(r2, static_cast<float>(qp - pos), 1.0f)), x);
          y = fmaf(-r1, __log2f(fmaf(r2, static_cast<float>(qp - pos - 1), 1.0f)), y);
        }
        if (!whole) {
          auto valid = [&](int p) {
            return t < kept_tiles ? p < kept : p <= qp && p >= lo && (a.window == 0 || p > qp - a.window || p < a.keep_first);
          };
          if (!valid(pos)) x = -INFINITY;
          if (!valid(pos + 1)) y = -INFINITY;
        }
        *reinterpret_cast<float2*>(at + lane_final) = make_float2(x, y);
      };
      if (a.score_mix != nullptr) {
#pragma unroll
        for (int j0 = 0; j0 < PIECES; j0 += AT_ONCE) {
          if (tok_first + j0 * TOKENS >= n_tok) break;           // (the same for the whole warp, as are the tokens below)
          float* at[AT_ONCE];
          unsigned hi3[AT_ONCE][HM / 16][2], mid3[AT_ONCE][HM / 16][2], low3[AT_ONCE][HM / 16][2];
#pragma unroll
          for (int u = 0; u < AT_ONCE; ++u) {
            // (a token past the last one has scores of whatever lies there, which nobody reads)
            at[u] = s_s + min(tok_first + (j0 + u) * TOKENS, NTOK - 1) * SST + key8;
#pragma unroll
            for (int kk = 0; kk < HM / 16; ++kk)
#pragma unroll
              for (int half = 0; half < 2; ++half) {
                const float* raw = at[u] + (kk * 16 + half * 8) * HST + lane_raw;
                ah_split(raw[0], raw[HST], hi3[u][kk][half], mid3[u][kk][half], low3[u][kk][half]);
              }
          }
          __syncwarp();                              // the raw scores of these keys are read
#pragma unroll
          for (int mt = 0; mt < HM / 16; ++mt) {
            float c[AT_ONCE][4];
#pragma unroll
            for (int u = 0; u < AT_ONCE; ++u) c[u][0] = c[u][1] = c[u][2] = c[u][3] = 0.0f;
#pragma unroll
            for (int kk = 0; kk < HM / 16; ++kk) {
              const unsigned m_at = mix_at + static_cast<unsigned>(mt * 16 * MST + kk * 16) * 2u;
              unsigned m[4];
              if (!one_part) {                       // the smaller products first
                ah_ldmatrix(m, m_at + 2u * (2 * HM * MST));
#pragma unroll
                for (int u = 0; u < AT_ONCE; ++u) mma_bf16_16816(c[u], m, hi3[u][kk][0], hi3[u][kk][1]);
                ah_ldmatrix(m, m_at + 2u * (HM * MST));
#pragma unroll
                for (int u = 0; u < AT_ONCE; ++u) {
                  mma_bf16_16816(c[u], m, mid3[u][kk][0], mid3[u][kk][1]);
                  mma_bf16_16816(c[u], m, hi3[u][kk][0], hi3[u][kk][1]);
                }
              }
              ah_ldmatrix(m, m_at);
#pragma unroll
              for (int u = 0; u < AT_ONCE; ++u) mma_bf16_16816(c[u], m, low3[u][kk][0], low3[u][kk][1]);
#pragma unroll
              for (int u = 0; u < AT_ONCE; ++u) mma_bf16_16816(c[u], m, mid3[u][kk][0], mid3[u][kk][1]);
#pragma unroll
              for (int u = 0; u < AT_ONCE; ++u) mma_bf16_16816(c[u], m, hi3[u][kk][0], hi3[u][kk][1]);
            }
#pragma unroll
            for (int u = 0; u < AT_ONCE; ++u) {
              const int tok = tok_first + (j0 + u) * TOKENS, h = mt * 16 + quad_row;
              if (tok < n_tok) {
                if (h < a.nh) finish(at[u] + mt * 16 * HST, tok, h, c[u][0], c[u][1]);
                if (h + 8 < a.nh) finish(at[u] + (mt * 16 + 8) * HST, tok, h + 8, c[u][2], c[u][3]);
              }
            }
          }
        }
      } else {
        for (int tok = tok_first; tok < n_tok; tok += TOKENS) {
          float* at = s_s + tok * SST + key8;
#pragma unroll
          for (int h8 = 0; h8 < HM; h8 += 8) {
            if (h8 + quad_row < a.nh) {
              const float2 raw = *reinterpret_cast<const float2*>(at + h8 * HST + lane_final);
              finish(at + h8 * HST, tok, h8 + quad_row, raw.x, raw.y);
            }
          }
        }
      }
    }
    cp_async_wait<1>();
    __syncthreads();                                 // the scores are final, this tile's values have landed
    // ------------------------------------------------------------------------------ softmax and values
    if (works) {
      unsigned pb[HPW][NT][MT][2];
#pragma unroll
      for (int i = 0; i < HPW; ++i) {
#pragma unroll
        for (int nt = 0; nt < NT; ++nt) {
          float2 v[BK / 8];
          float top = -INFINITY;
          const bool real = head0 + i < a.nh;        // (uniform over the warp)
#pragma unroll
          for (int j = 0; j < BK / 8; ++j) {
            v[j] = real ? *reinterpret_cast<const float2*>(own_at + i * HST + nt * 8 * SST + 8 * j) : make_float2(0.0f, 0.0f);
            top = fmaxf(top, fmaxf(v[j].x, v[j].y));
          }
          top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, 1));
          top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, 2));
          const float new_m = fmaxf(m_run[i][nt], top);
          const float m_use = new_m == -INFINITY ? 0.0f : new_m;      // a token that has seen no key yet
          const float corr = ah_exp2(m_run[i][nt] - m_use);
          m_run[i][nt] = new_m;
          float sum = 0.0f;
#pragma unroll
          for (int j = 0; j < BK / 8; ++j) {
            v[j].x = ah_exp2(v[j].x - m_use);
            v[j].y = ah_exp2(v[j].y - m_use);
            sum += v[j].x + v[j].y;
          }
          sum += __shfl_xor_sync(0xffffffffu, sum, 1);
          sum += __shfl_xor_sync(0xffffffffu, sum, 2);
          l_run[i][nt] = l_run[i][nt] * corr + sum;
#pragma unroll
          for (int ks = 0; ks < MT; ++ks) {
            pb[i][nt][ks][0] = pack_bf16(v[2 * ks].x, v[2 * ks].y);
            pb[i][nt][ks][1] = pack_bf16(v[2 * ks + 1].x, v[2 * ks + 1].y);
          }
          if (!__all_sync(0xffffffffu, corr == 1.0f)) {               // tokens 2 quad and 2 quad + 1 own this lane's columns
            const float c0 = __shfl_sync(0xffffffffu, corr, 8 * quad), c1 = __shfl_sync(0xffffffffu, corr, 8 * quad + 4);
#pragma unroll
            for (int m = 0; m < DM; ++m) {
              o[i][nt][m][0] *= c0; o[i][nt][m][1] *= c1; o[i][nt][m][2] *= c0; o[i][nt][m][3] *= c1;
            }
          }
        }
      }
#pragma unroll
      for (int m = 0; m < DM; ++m) {
        if (m < vm_n) {
#pragma unroll
          for (int i = 0; i < HPW; ++i) {
#pragma unroll
            for (int ks = 0; ks < MT; ++ks) {
              unsigned va[4];
              ah_ldmatrix_trans(va, v_at[i] + ks * v_step + m * 32);
#pragma unroll
              for (int nt = 0; nt < NT; ++nt) mma_bf16_16816(o[i][nt][m], va, pb[i][nt][ks][0], pb[i][nt][ks][1]);
            }
          }
        }
      }
    }
    cp_async_wait<0>();
    __syncthreads();                                 // the next keys have landed; scores and values are read
    if (more) load_values(buffer ^ 1);
    cp_async_commit();
  }
  cp_async_wait<0>();

#pragma unroll
  for (int i = 0; i < HPW; ++i) {
    const int head = head0 + i;
    if (head >= a.nh || col0 >= n_tok) break;
    if (a.splits > 1) {                              // one token: column 0 of the first tokens' column
      const size_t slot = (static_cast<size_t>(tile) * a.splits + split) * a.nh + head;
      if (lane == 0) {
        a.part_ml[2 * slot] = m_run[i][0];
        a.part_ml[2 * slot + 1] = l_run[i][0];
      }
      if (quad == 0) {
#pragma unroll
        for (int m = 0; m < DM; ++m) {
          const int d = m * 16 + quad_row;
          if (d < a.vd) a.part_o[slot * a.vd + d] = o[i][0][m][0];
          if (d + 8 < a.vd) a.part_o[slot * a.vd + d + 8] = o[i][0][m][2];
        }
      }
      continue;
    }
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) {
      const float l0 = __shfl_sync(0xffffffffu, l_run[i][nt], 8 * quad), l1 = __shfl_sync(0xffffffffu, l_run[i][nt], 8 * quad + 4);
      const float inv[2] = {l0 > 0.0f ? 1.0f / l0 : 0.0f, l1 > 0.0f ? 1.0f / l1 : 0.0f};
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const int tok = col0 + nt * 8 + 2 * quad + u;
        if (tok >= n_tok) continue;
        __nv_bfloat16* dst = a.out + (static_cast<size_t>(tok0 + tok) * a.nh + head) * a.vd;
#pragma unroll
        for (int m = 0; m < DM; ++m) {
          const int d = m * 16 + quad_row;
          if (d < a.vd) dst[d] = __float2bfloat16_rn(o[i][nt][m][u] * inv[u]);
          if (d + 8 < a.vd) dst[d + 8] = __float2bfloat16_rn(o[i][nt][m][2 + u] * inv[u]);
        }
      }
    }
  }
}

// The splits' partial results of one token and head, in the order of the context.
constexpr int AH_MERGE_THREADS = 128;
constexpr int AH_MAX_SPLITS = AH_MERGE_THREADS;      // a thread each

__global__ void __launch_bounds__(AH_MERGE_THREADS) heads_merge_kernel(const HeadsAttentionArgs a) {
  __shared__ float weight_s[AH_MAX_SPLITS];
  __shared__ float warp_note[AH_MERGE_THREADS / 32];
  __shared__ float scratch[33];
  const int tile = blockIdx.x, head = blockIdx.y, split = threadIdx.x;
  const int row = a.tile_row[tile];
  if (row < 0 || row >= a.num_rows || a.row_q_len[row] - a.tile_q0[tile] <= 0) return;       // (reported by the other kernel)
  const size_t slot0 = static_cast<size_t>(tile) * a.splits * a.nh + head;
  float m = -INFINITY, l = 0.0f;
  if (split < a.splits) {
    const float2 ml = *reinterpret_cast<const float2*>(a.part_ml + 2 * (slot0 + static_cast<size_t>(split) * a.nh));
    m = ml.x;
    l = ml.y;
  }
  const float warp_top = warp_max(m);
  if ((threadIdx.x & 31) == 0) warp_note[threadIdx.x >> 5] = warp_top;
  __syncthreads();
  float top = warp_note[0];
#pragma unroll
  for (int i = 1; i < AH_MERGE_THREADS / 32; ++i) top = fmaxf(top, warp_note[i]);
  const float weight = m > -INFINITY ? exp2f(m - top) : 0.0f;
  weight_s[split] = weight;
  const float sum = block_sum(l * weight, scratch);  // (a barrier: the weights are there)
  const float inv = sum > 0.0f ? 1.0f / sum : 0.0f;
  const size_t token = a.row_q_start[row] + a.tile_q0[tile];
  for (int d = threadIdx.x; d < a.vd; d += AH_MERGE_THREADS) {
    float v = 0.0f;
#pragma unroll 8
    for (int s = 0; s < a.splits; ++s) v = fmaf(a.part_o[(slot0 + static_cast<size_t>(s) * a.nh) * a.vd + d], weight_s[s], v);
    a.out[(token * a.nh + head) * a.vd + d] = __float2bfloat16_rn(v * inv);
  }
}

struct HeadsShape {
  int warps, hpw, nt, cg, dm, bk;
  size_t smem;
};

// How the kernel runs this layer (warps 0: it does not take it); `single`: for tiles of one token.
HeadsShape heads_shape(int nh, int nkv, int kd, int vd, bool single) {
  HeadsShape shape{0, 0, 0, 0, 0, 0, 0};
  if (nh <= 0 || nkv <= 0 || nh % nkv != 0 || kd <= 0 || vd <= 0) return shape;
  const int widest = (kd > vd ? kd : vd);
  const int dm = widest <= 64 ? 4 : (widest <= 128 ? 8 : (widest <= 256 ? 16 : 0));
  const int hpw = nh <= 16 ? 1 : (nh <= 32 ? 2 : 0);
  if (dm == 0 || hpw == 0 || (dm == 16 && hpw == 2)) return shape;
  // Up to 8 heads: eight warps for a token, sixteen in two column groups for a prompt.
  const int cg = nh <= 8 && !single ? 2 : 1, warps = nh <= 8 && single ? 8 : 16;
  const int nt = single || nh <= 8 || hpw == 2 || dm == 16 ? 1 : 2;
  const int hm = nh <= 16 ? 16 : 32;
  for (int bk = 32; bk >= 16; bk -= 16) {
    const size_t smem = static_cast<size_t>(nkv) * bk * (ah_padded(kd) + ah_padded(vd)) * sizeof(__nv_bfloat16) +
                        static_cast<size_t>(3) * hm * (hm + 8) * sizeof(__nv_bfloat16) +
                        static_cast<size_t>(hm) * ah_head_stride(8 * nt * cg, bk) * sizeof(float);
    if (smem + 2048 <= AH_SMEM_LIMIT) {
      shape = HeadsShape{warps, hpw, nt, cg, dm, bk, smem};
      return shape;
    }
  }
  return shape;
}

template <int W, int HPW, int NT, int CG, int DM, int BK>
int heads_launch(const HeadsAttentionArgs& a, int n_tiles, size_t smem, cudaStream_t stream) {
  auto kernel = heads_attention_kernel<W, HPW, NT, CG, DM, BK>;
  if (cuda_failed(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)))) return ERR_CUDA;
  kernel<<<dim3(a.splits, n_tiles), W * 32, smem, stream>>>(a);
  return launch_result();
}

}  // namespace zb

using namespace zb;

// New tokens of one request that a tile covers for rows with several of them (0: the shape is not taken).
ZB_API int zb_heads_attention_tile_tokens(int nh, int nkv, int kd, int vd, int dtype) {
  if (dtype != DTYPE_BF16) return 0;
  if (heads_shape(nh, nkv, kd, vd, true).warps == 0) return 0;
  const HeadsShape shape = heads_shape(nh, nkv, kd, vd, false);
  return shape.warps == 0 ? 0 : 8 * shape.nt * shape.cg;
}

// Keys of a tile of a decoded token: its keys can be cut into at most ceil(keys / this) splits that all have work.
ZB_API int zb_heads_attention_tile_keys(int nh, int nkv, int kd, int vd) { return heads_shape(nh, nkv, kd, vd, true).bk; }

// Attention of the tiles' tokens over their requests' pages; writes those tokens' rows of `out` [T, nh * vd].
// `single`: every tile is one token, whose keys `splits` CTAs share; with splits > 1 `scratch` holds
// n_tiles * splits * nh * (vd + 2) floats (contents irrelevant); at most 128 splits.
ZB_API int zb_heads_attention(void* out, const void* q, const void* kv_cache, const int* block_table, int max_blocks,
                              int page_size, int num_pages, int num_rows, const int* tile_row, const int* tile_q0,
                              int n_tiles, const int* row_q_start, const int* row_q_len, const int* row_ctx, int nh,
                              int nkv, int kd, int vd, int window, int keep_first, float scale, const float* score_mix,
                              const float* bias_r1, const float* bias_r2, const float* sinks, int single, int splits, float* scratch,
                              int* status, void* stream) {
  if (n_tiles < 0 || page_size <= 0 || window < 0 || keep_first < 0 || splits <= 0 || splits > AH_MAX_SPLITS || (splits > 1 && (!single || scratch == nullptr)) ||
      (bias_r1 == nullptr) != (bias_r2 == nullptr) || reinterpret_cast<uintptr_t>(q) % 4 != 0 ||
      reinterpret_cast<uintptr_t>(kv_cache) % 16 != 0)
    return ERR_BAD_ARGUMENT;
  const HeadsShape shape = heads_shape(nh, nkv, kd, vd, single != 0);
  if (shape.warps == 0) return ERR_UNSUPPORTED;
  if (n_tiles == 0) return OK;
  if (n_tiles > 65535) return ERR_UNSUPPORTED;
  HeadsAttentionArgs a;
  a.q = static_cast<const __nv_bfloat16*>(q);
  a.out = static_cast<__nv_bfloat16*>(out);
  a.kv_cache = static_cast<const __nv_bfloat16*>(kv_cache);
  a.block_table = block_table; a.tile_row = tile_row; a.tile_q0 = tile_q0;
  a.row_q_start = row_q_start; a.row_q_len = row_q_len; a.row_ctx = row_ctx;
  a.max_blocks = max_blocks; a.page_size = page_size; a.num_pages = num_pages; a.num_rows = num_rows;
  a.page_shift = -1;
  for (int shift = 0; shift < 31; ++shift)
    if (page_size == (1 << shift)) a.page_shift = shift;
  a.nh = nh; a.nkv = nkv; a.kd = kd; a.vd = vd; a.window = window; a.keep_first = window > 0 ? keep_first : 0;
  a.scale_log2 = scale * 1.4426950408889634f;
  a.score_mix = score_mix; a.bias_r1 = bias_r1; a.bias_r2 = bias_r2; a.sinks = sinks;
  a.splits = splits;
  a.part_ml = scratch;                               // pairs of floats first: they stay on 8-byte boundaries
  a.part_o = scratch != nullptr ? scratch + static_cast<size_t>(n_tiles) * splits * nh * 2 : nullptr;
  a.status = status;
  auto s = static_cast<cudaStream_t>(stream);
  int rc = ERR_UNSUPPORTED;
#define ZB_AH(W, HPW, NT, CG, DM, BK)                                                                              \
  if (shape.warps == W && shape.hpw == HPW && shape.nt == NT && shape.cg == CG && shape.dm == DM && shape.bk == BK) \
    rc = heads_launch<W, HPW, NT, CG, DM, BK>(a, n_tiles, shape.smem, s);
#define ZB_AH_BK(W, HPW, NT, CG, DM) ZB_AH(W, HPW, NT, CG, DM, 32) ZB_AH(W, HPW, NT, CG, DM, 16)
  ZB_AH_BK(8, 1, 1, 1, 4) ZB_AH_BK(16, 1, 1, 2, 4) ZB_AH_BK(16, 1, 1, 1, 4) ZB_AH_BK(16, 1, 2, 1, 4) ZB_AH_BK(16, 2, 1, 1, 4)
  ZB_AH_BK(8, 1, 1, 1, 8) ZB_AH_BK(16, 1, 1, 2, 8) ZB_AH_BK(16, 1, 1, 1, 8) ZB_AH_BK(16, 1, 2, 1, 8) ZB_AH_BK(16, 2, 1, 1, 8)
  ZB_AH_BK(8, 1, 1, 1, 16) ZB_AH_BK(16, 1, 1, 2, 16) ZB_AH_BK(16, 1, 1, 1, 16)
#undef ZB_AH_BK
#undef ZB_AH
  if (rc != OK || splits == 1) return rc;
  heads_merge_kernel<<<dim3(n_tiles, nh), AH_MERGE_THREADS, 0, s>>>(a);
  return launch_result();
}
