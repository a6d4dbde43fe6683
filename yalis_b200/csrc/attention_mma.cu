// Paged causal attention on the tensor cores (bfloat16 in, float32 softmax and
// accumulation), one kernel for prompt portions, single decoded tokens and any
// mix of them.
//
// Work is cut by (request, KV head): all query heads that share a KV head and
// all tokens the request brings to this step form the rows of one problem,
// row = token * heads_per_group + head_in_group, so a K/V tile read from the
// cache serves every one of them (for a decode step that is the whole GQA group
// of one token).  A block takes 64 rows (4 warps x 16) and walks the visible
// keys in tiles of 64: K and V tiles are gathered page by page with cp.async
// into padded shared memory (double buffered), S = Q K^T and O += P V run on
// mma.sync.m16n8k16 with ldmatrix operand loads, the online softmax is kept in
// registers in the exp2 domain.  The mask is by absolute position: the row of a
// token at position p sees keys j with p - window < j <= p
// (yalis/attention/backend_impl/sdpa_and_flex.py:15-19, 301-307).
//
// When a (request, KV head) has at most 16 rows (a decode step: one token, up to 16 heads per
// group) the four warps do not own rows: all work on the same 16 rows and each takes a
// quarter of every key tile, and their four partial softmax states are merged through
// shared memory at the end.
//
// With n_splits > 1 (decode steps of few requests) the keys of a request are
// divided among blocks; each writes an unnormalised partial result with its
// running maximum and sum to scratch memory and takes a ticket from a counter of
// its (request, KV head); the block that draws the last ticket merges all splits
// in index order (so the result does not depend on which block came last) and
// resets the counter for the next launch.
//
// The general form (GEN) adds what some mixers ask of attention: scores squeezed by
// c * tanh(s / c), a sink (a key of score 0 and no value: 1 more in the denominator), a
// learned score of that sink per head, a chunked mask (a row sees only the keys of its own chunk of C positions),
// a distance bias slope_h * (pos - key) taken off the score, a sigmoid gate on the result,
// a factor on the result, and weights that meet V with 16 bits of mantissa instead of 8:
// P is split into its bfloat16 rounding and the bfloat16 rounding of the rest, and both
// halves go through the tensor cores (the sum of the weights is float32 in either form).
//
// The extended form (FORM 2 and 3) is the general form with head sizes that are known at launch only
// (keys and values may differ; both multiples of 8, padded to one of three tile widths), a
// learned bias per head and distance added to the scaled score, and pooled blocks: beside the
// keys of its window a row sees one key and value for every block of P positions that lies
// wholly before the window.  The blocks have pools and a block table of their own; their tiles
// come first, then those of the window, in one softmax.
//
// The form of two maps (FORM 4 and 5) has two queries per head and two keys per key/value head and position (side by side in a
// cached row of 2 d sizes) over one value: each map is a softmax of its own, and the result is the first map's minus
// lambda times the second's, divided by its root mean square, times a factor.  A row is then a (token, head, map): a
// block takes half as many pairs (token, head) as it has rows, the first half of its rows for the first map and the second
// half for the second, so a K tile of 2 d columns and its V tile are read once for both.  In prompts a warp's rows belong
// to one map and it multiplies only that map's half of the columns; in decode steps the rows of both maps share a
// warp and a row's query is zero in the other map's half.  The maps meet in shared memory, in float32, at the end.
#include "common.cuh"

namespace {

constexpr int BM = 64;   // rows per block
constexpr int BN = 64;   // keys per tile
constexpr int NWARPS = 4;

struct AttnParams {
  const __nv_bfloat16* q;      // [N, q_stride], head h at column h*HS
  int q_stride;
  __nv_bfloat16* out;          // [N, out_stride]
  int out_stride;
  const __nv_bfloat16* k_pool; // [pages, g, page_size, HS]
  const __nv_bfloat16* v_pool;
  const int32_t* positions;    // [N]
  const int32_t* q_start;      // [R+1]
  const int32_t* block_table;  // [R, table_width]
  int table_width, page_size, num_pages;
  int page_shift;              // log2(page_size) if it is a power of two, else -1
  int nh, g, per;              // per = nh / g
  float scale_log2;            // scale * log2(e)
  float cap_log2;              // GEN: soft cap * log2(e) (0: no cap)
  float scale_over_cap;        // GEN: scale / soft cap
  int sink;                    // GEN: 1 adds exp(0) to every row's denominator
  float out_scale;             // GEN: factor on the result
  int exact_weights;           // ask for the general form even without cap, sink or factor
  int window;                  // 0: none
  int chunk;                   // GEN: C > 0: a row at position p sees keys >= floor(p / C) * C only
  const float* sink_logits;    // GEN: [nh] score of the sink per head (null: 0)
  const float* slopes;         // GEN: [nh] slope_h * (p - key) is taken off the score (null: none)
  const __nv_bfloat16* gate;   // GEN: [N, gate_stride] the result is multiplied by sigmoid(gate[t, head, :]) (null: not)
  int gate_stride;
  int gate_per_head;           // GEN: the gate is [N, nh], one number per head
  int map_dim;                 // FORM 4, 5: d, the size of one map's query and key (hs = 2 d, a multiple of 32)
  float lambda, diff_eps;      // FORM 4, 5
  int hs, vs;                  // FORM 2, 3, 4: sizes of a key and a value (multiples of 8, at most HS)
  const float* rel;            // FORM 2, 3: [nh, rel_len], rel[h][min(p - key, rel_len - 1)] is added to the scaled score (null: not)
  int rel_len;
  int rel_staged;              // the table of a block's heads fits the shared memory set aside for it
  int pool;                    // FORM 2, 3: P > 0: pooled blocks of P positions before the window
  const __nv_bfloat16* pk_pool; const __nv_bfloat16* pv_pool;   // [pages, g, pool_page_size, HS / VS], an entry per block
  const int32_t* pool_table;
  int pool_table_width, pool_page_size, pool_num_pages, pool_page_shift;
  int n_splits;
  float* part_o;               // [N, nh, n_splits, HS] (split mode); FORM 4, 5: [N, nh, 2, n_splits, HS]
  float* part_ml;              // the same places, 2 floats each
  int32_t* tickets;            // one per block of a split: zero before the launch and zero again after it (split mode)
};

__device__ __forceinline__ void cp_async16(void* smem, const void* gmem) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(s), "l"(gmem));
}
// The same, or 16 zero bytes (nothing is read then, but `gmem` must be an address of the pool).
__device__ __forceinline__ void cp_async16_or_zero(void* smem, const void* gmem, bool copy) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(s), "l"(gmem), "r"(copy ? 16 : 0));
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;\n" ::); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N)); }

__device__ __forceinline__ void ldmatrix_x4(unsigned (&r)[4], const void* smem) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(s));
}
__device__ __forceinline__ void ldmatrix_x4_trans(unsigned (&r)[4], const void* smem) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(s));
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ unsigned pack_bf16(float lo, float hi) {
  __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<unsigned*>(&v);
}

// Gathers keys [key0, key0 + BN) of one KV head into two [BN][HS + 8] tiles (K and V); rows
// outside [lo_key, hi_key] or on an unmapped page are zero-filled.  Consecutive threads copy
// consecutive 16-byte chunks of a row (coalesced); all page lookups of a thread are done
// before its first copy is issued, so that they overlap.
template <int HS>
__device__ __forceinline__ void load_kv_tile(__nv_bfloat16* k_dst, __nv_bfloat16* v_dst, const int32_t* bt,
                                             const AttnParams& p, int kvh, int key0, int lo_key, int hi_key) {
  constexpr int CHUNKS = HS / 8;                          // 16-byte chunks per row
  constexpr int LD = HS + 8;
  constexpr int ITERS = BN * CHUNKS / (NWARPS * 32);      // chunks per thread (HS % 16 == 0 makes it whole)
  static_assert(BN * CHUNKS % (NWARPS * 32) == 0, "tile chunks must divide among the threads");
  long long src[ITERS];
  const int head_stride = p.page_size * HS;               // elements of one (page, kv head) block
#pragma unroll
  for (int i = 0; i < ITERS; ++i) {
    const int c = threadIdx.x + i * (NWARPS * 32);
    const int row = c / CHUNKS, ch = c - row * CHUNKS;
    const int key = key0 + row;
    src[i] = -1;
    if (key >= lo_key && key <= hi_key) {
      const int pi = p.page_shift >= 0 ? (key >> p.page_shift) : (key / p.page_size);
      const int page = pi < p.table_width ? bt[pi] : -1;
      if (page >= 0 && page < p.num_pages)
        src[i] = (long long)(page * p.g + kvh) * head_stride + (key - pi * p.page_size) * HS + ch * 8;
    }
  }
#pragma unroll
  for (int i = 0; i < ITERS; ++i) {
    const int c = threadIdx.x + i * (NWARPS * 32);
    const int row = c / CHUNKS, ch = c - row * CHUNKS;
    __nv_bfloat16* kd = k_dst + row * LD + ch * 8;
    __nv_bfloat16* vd = v_dst + row * LD + ch * 8;
    if (src[i] >= 0) {
      cp_async16(kd, p.k_pool + src[i]);
      cp_async16(vd, p.v_pool + src[i]);
    } else {
      *reinterpret_cast<uint4*>(kd) = make_uint4(0u, 0u, 0u, 0u);
      *reinterpret_cast<uint4*>(vd) = make_uint4(0u, 0u, 0u, 0u);
    }
  }
}

// The same for the extended form: keys and values of sizes known at launch, columns past them zero, from the token
// pages or (`pooled`) from the pages of the pooled blocks.
template <int HS, bool SIZED>
__device__ __forceinline__ void load_kv_tile_extended(__nv_bfloat16* k_dst, __nv_bfloat16* v_dst, const AttnParams& p, int req,
                                                   int kvh, int key0, int lo_key, int hi_key, bool pooled) {
  constexpr int CHUNKS = HS / 8, LD = HS + 8;
  const int width = pooled ? p.pool_table_width : p.table_width;
  const int32_t* bt = (pooled ? p.pool_table : p.block_table) + (size_t)req * width;
  const int shift = pooled ? p.pool_page_shift : p.page_shift;
  const int ps = pooled ? p.pool_page_size : p.page_size, pages = pooled ? p.pool_num_pages : p.num_pages;
  const __nv_bfloat16* kp = pooled ? p.pk_pool : p.k_pool;
  const __nv_bfloat16* vp = pooled ? p.pv_pool : p.v_pool;
  constexpr int ITERS = BN * CHUNKS / (NWARPS * 32);
  static_assert(BN * CHUNKS % (NWARPS * 32) == 0, "tile chunks must divide among the threads");
  long long at[ITERS];                                    // row of the pool, -1: none
#pragma unroll
  for (int i = 0; i < ITERS; ++i) {
    const int c = threadIdx.x + i * (NWARPS * 32);
    const int key = key0 + c / CHUNKS;
    at[i] = -1;
    if (key >= lo_key && key <= hi_key) {
      const int pi = shift >= 0 ? (key >> shift) : (key / ps);
      const int page = pi < width ? bt[pi] : -1;
      if (page >= 0 && page < pages) at[i] = ((long long)page * p.g + kvh) * ps + (key - pi * ps);
    }
  }
#pragma unroll
  for (int i = 0; i < ITERS; ++i) {
    const int c = threadIdx.x + i * (NWARPS * 32);
    const int row = c / CHUNKS, ch = c - row * CHUNKS;
    __nv_bfloat16* kd = k_dst + row * LD + ch * 8;
    __nv_bfloat16* vd = v_dst + row * LD + ch * 8;
    const bool row_ok = at[i] >= 0;
    const long long r = row_ok ? at[i] : 0;
    const int hs = SIZED ? p.hs : HS, vs = SIZED ? p.vs : HS;
    const bool k_ok = row_ok && (!SIZED || ch * 8 < hs), v_ok = row_ok && (!SIZED || ch * 8 < vs);
    cp_async16_or_zero(kd, kp + (k_ok ? r * hs + ch * 8 : 0), k_ok);
    cp_async16_or_zero(vd, vp + (v_ok ? r * vs + ch * 8 : 0), v_ok);
  }
}

// DEC: the block has at most 16 rows; warps split the keys of a tile instead of the rows.
// A score in the exp2 domain: s * scale * log2(e), or with a cap c: c * tanh(s * scale / c) * log2(e).
// `bias_log2`: what is taken off the scaled score before the cap, in the exp2 domain (the distance bias).
template <bool GEN>
__device__ __forceinline__ float score_log2(const AttnParams& p, float s, float bias_log2 = 0.f) {
  if (GEN && p.cap_log2 > 0.f) {
    // tanh(x) = 1 - 2 / (exp(2x) + 1) with the fast exponential and reciprocal: absolute error about 3e-7, which
    // the cap multiplies to 1e-5 of a score at most (the float32 path uses tanhf in the exact kernel)
    const float x = fminf(s * p.scale_over_cap - bias_log2 / p.cap_log2, 15.f);
    return p.cap_log2 * (1.0f - __fdividef(2.0f, __expf(2.0f * x) + 1.0f));
  }
  return GEN ? s * p.scale_log2 - bias_log2 : s * p.scale_log2;
}

// The sink's score of a head in the exp2 domain.
__device__ __forceinline__ float sink_log2(const AttnParams& p, int head) {
  return p.sink_logits ? p.sink_logits[head] * 1.4426950408889634f : 0.f;
}
// sigmoid of the gate that belongs to out[tok, head, d].
__device__ __forceinline__ float gate_factor(const AttnParams& p, int tok, int head, int hs, int d) {
  const size_t at = (size_t)tok * p.gate_stride + (p.gate_per_head ? (size_t)head : (size_t)head * hs + d);
  return 1.0f / (1.0f + __expf(-__bfloat162float(p.gate[at])));
}
// The first key a row at position `pos` sees.
template <bool GEN>
__device__ __forceinline__ int first_visible(const AttnParams& p, int pos) {
  int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0;
  if (GEN && p.chunk > 0) lo = max(lo, (pos / p.chunk) * p.chunk);
  return lo;
}

// How many pooled blocks a row at position `pos` sees: those that end at or before pos - window.
__device__ __forceinline__ int blocks_seen(const AttnParams& p, int pos) {
  return (p.pool > 0 && pos - p.window + 1 > 0) ? (pos - p.window + 1) / p.pool : 0;
}

// Normalisation of a finished row: with a sink the denominator gains exp2(0 - m) for the row's maximum m
// (the maximum itself is raised to 0 first when all scores lie below it).
template <bool GEN>
__device__ __forceinline__ float finish_factor(const AttnParams& p, float m, float l, float sink_z = 0.f) {
  if (GEN && p.sink) {
    // numerator and denominator are relative to exp2(m): the sink is exp2(z - m) in that unit
    l += exp2f(sink_z - m);
    return p.out_scale / l;
  }
  return l > 0.f ? (GEN ? p.out_scale : 1.0f) / l : 0.f;
}

// FORM: 0 plain, 1 general, 2 extended, 3 extended with sizes known at launch (HS is then the padded size; p.hs and p.vs
// are the real ones), 4 two maps (sizes known at launch too; p.hs is that of both maps' keys together), 5 two maps whose
// keys together and values both have size HS.
template <int HS, bool DEC, int FORM>
__global__ void __launch_bounds__(NWARPS * 32) paged_attention_mma_kernel(const AttnParams p) {
  constexpr bool GEN = FORM >= 1, EXT = FORM >= 2 && FORM <= 4, SIZED = FORM == 3 || FORM == 4, MAPS = FORM >= 4;
  const int hs = SIZED ? p.hs : HS, vs = SIZED ? p.vs : HS;
  constexpr int LD = HS + 8;            // padded row: ldmatrix rows fall into distinct banks
  constexpr int KSTEPS = HS / 16;       // k-steps of Q K^T
  constexpr int DT = HS / 8;            // n8 tiles of the output along the head dimension
  constexpr int WKEYS = DEC ? BN / NWARPS : BN;   // keys of a tile that one warp handles
  constexpr int ST = WKEYS / 8;         // n8 tiles of S along this warp's keys
  constexpr int RB = DEC ? 16 : BM;     // rows per block
  constexpr int PB = MAPS ? RB / 2 : RB;            // pairs (token, head) per block: rows r and r + PB are the maps of one
  constexpr bool HALF = MAPS && !DEC;               // a warp multiplies one map's half of the columns
  constexpr int QSTEPS = HALF ? KSTEPS / 2 : KSTEPS;
  constexpr int NST = DEC ? 3 : 2;      // K/V tiles in flight: decode blocks are latency bound
  extern __shared__ __align__(16) unsigned char smem_raw[];
  __nv_bfloat16* q_s = reinterpret_cast<__nv_bfloat16*>(smem_raw);   // [RB][LD]
  __nv_bfloat16* k_s = q_s + RB * LD;                                 // [NST][BN][LD]
  __nv_bfloat16* v_s = k_s + NST * BN * LD;                           // [NST][BN][LD]
  float* rel_s = reinterpret_cast<float*>(v_s + NST * BN * LD);       // extended: [per][rel_len] in the exp2 domain
  pdl_launch_dependents();
  pdl_wait();

  const int req = blockIdx.y / p.g, kvh = blockIdx.y - req * p.g;
  const int tok0 = p.q_start[req], q_len = p.q_start[req + 1] - tok0;
  const int n_rows = q_len * p.per;              // (two maps: pairs)
  const int row0 = blockIdx.x * PB;
  if (row0 >= n_rows) return;
  const int split = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int gid = lane >> 2, tig = lane & 3;
  const int wrow = DEC ? 0 : warp * 16;           // first row of this warp within the block's tile
  const int wkey = DEC ? warp * WKEYS : 0;        // first key of this warp within a key tile
  const int wcol = HALF ? (wrow / PB) * p.map_dim : 0;         // first column of this warp's queries and keys
  const int wcols = HALF ? p.map_dim : hs;        // (looked at where sizes are known at launch)
  const int32_t* bt = p.block_table + (size_t)req * p.table_width;

  // Positions of the tile's first and last token bound the keys this block needs.
  const int first_tok = row0 / p.per;
  const int last_row = min(row0 + PB, n_rows) - 1;
  const int last_tok = last_row / p.per;
  const int pos_first = p.positions[tok0 + first_tok];
  const int pos_last = p.positions[tok0 + last_tok];
  const int lo_key = first_visible<GEN>(p, pos_first);      // positions grow along a portion: the smallest bound
  const int lo_last = first_visible<GEN>(p, pos_last);      // and the largest
  const int hi_key = pos_last;
  int tile_lo = lo_key / BN, tile_hi = hi_key / BN + 1;     // key tiles [tile_lo, tile_hi)
  if (p.n_splits > 1) {
    const int total = tile_hi - tile_lo;
    const int per_split = (total + p.n_splits - 1) / p.n_splits;
    tile_lo = tile_lo + split * per_split;
    tile_hi = min(tile_hi, tile_lo + per_split);
  }
  // Extended form: the tiles of the pooled blocks come first, `pool_tiles` of them; tile v < pool_tiles holds blocks
  // [v * BN, ...), tile v >= pool_tiles the keys of tile first_key_tile + v - pool_tiles.
  int pool_tiles = 0, first_key_tile = tile_lo, nb_last = 0;
  if (EXT) {
    first_key_tile = lo_key / BN;
    nb_last = blocks_seen(p, pos_last);
    pool_tiles = (nb_last + BN - 1) / BN;
    const int total = pool_tiles + hi_key / BN + 1 - first_key_tile;
    const int per_split = (total + p.n_splits - 1) / p.n_splits;
    tile_lo = split * per_split;
    tile_hi = min(total, tile_lo + per_split);
  }
  const int n_tiles = max(0, tile_hi - tile_lo);
  auto load_tile = [&](int buf, int tile) {       // tile: counted from the block's first (extended: over both kinds)
    __nv_bfloat16* kd = k_s + buf * BN * LD;
    __nv_bfloat16* vd = v_s + buf * BN * LD;
    if constexpr (EXT) {
      if (tile < pool_tiles) load_kv_tile_extended<HS, SIZED>(kd, vd, p, req, kvh, tile * BN, 0, nb_last - 1, true);
      else load_kv_tile_extended<HS, SIZED>(kd, vd, p, req, kvh, (first_key_tile + tile - pool_tiles) * BN, lo_key, hi_key, false);
    } else {
      load_kv_tile<HS>(kd, vd, bt, p, kvh, tile * BN, lo_key, hi_key);
    }
  };

  // ---- Q tile -> shared memory, then this warp's A fragments ----------------------
  {
    constexpr int CHUNKS = HS / 8;
    for (int c = threadIdx.x; c < RB * CHUNKS; c += NWARPS * 32) {
      const int r = c / CHUNKS, ch = c - r * CHUNKS;
      const int row = row0 + r % PB;
      __nv_bfloat16* d = q_s + r * LD + ch * 8;
      bool mine = !SIZED || ch * 8 < hs;
      if (MAPS) mine = mine && (ch * 8 >= p.map_dim) == (r >= PB);    // the other map's half of the row stays zero
      if (row < n_rows && mine) {
        const int t = row / p.per, h = row - t * p.per;
        cp_async16(d, p.q + (size_t)(tok0 + t) * p.q_stride + (size_t)(kvh * p.per + h) * hs + ch * 8);
      } else {
        *reinterpret_cast<uint4*>(d) = make_uint4(0u, 0u, 0u, 0u);
      }
    }
  }
  if (EXT && p.rel && p.rel_staged) {
    const float* src = p.rel + (size_t)kvh * p.per * p.rel_len;
    for (int e = threadIdx.x; e < p.per * p.rel_len; e += NWARPS * 32) rel_s[e] = src[e] * 1.4426950408889634f;
  }
  // Prologue: Q and the first tile form one group, then NST-2 further tiles one group each.
#pragma unroll
  for (int t = 0; t < NST - 1; ++t) {
    if (t < n_tiles) load_tile(t, tile_lo + t);
    cp_async_commit();
  }
  cp_async_wait<NST - 2>();     // the group with Q and tile 0 has landed
  __syncthreads();

  unsigned qf[QSTEPS][4];
#pragma unroll
  for (int ks = 0; ks < QSTEPS; ++ks) {
    const int r = wrow + (lane & 7) + ((lane >> 3) & 1) * 8;
    const int c = wcol + ks * 16 + (lane >> 4) * 8;
    ldmatrix_x4(qf[ks], q_s + r * LD + c);
  }
  // Rows of this thread: gid and gid + 8 of the warp's 16.
  int row_pos[2], row_lo[2];
  bool row_ok[2];
  float row_slope[2] = {0.f, 0.f};      // in the exp2 domain
  int row_blocks[2] = {0, 0};           // extended: pooled blocks the row sees
  const float* row_rel[2] = {nullptr, nullptr};
  int row_head[2] = {0, 0};
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int row = row0 + (wrow + gid + i * 8) % PB;
    row_ok[i] = row < n_rows;
    row_pos[i] = row_ok[i] ? p.positions[tok0 + row / p.per] : -1;
    row_lo[i] = row_ok[i] ? first_visible<GEN>(p, row_pos[i]) : 0;
    if (GEN && p.slopes && row_ok[i]) row_slope[i] = p.slopes[kvh * p.per + row % p.per] * 1.4426950408889634f;
    if (EXT && row_ok[i]) {
      row_blocks[i] = blocks_seen(p, row_pos[i]);
      row_head[i] = row % p.per;
      if (p.rel) row_rel[i] = p.rel + (size_t)(kvh * p.per + row % p.per) * p.rel_len;
    }
  }
  const int nb_first = EXT ? blocks_seen(p, pos_first) : 0;

  float o[DT][4];
#pragma unroll
  for (int d = 0; d < DT; ++d) o[d][0] = o[d][1] = o[d][2] = o[d][3] = 0.f;
  float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};

  for (int it = 0; it < n_tiles; ++it) {
    const int buf = it % NST;
    const bool pooled = EXT && tile_lo + it < pool_tiles;
    const int key0 = (EXT && !pooled ? first_key_tile - pool_tiles + tile_lo + it : tile_lo + it) * BN;
    // prefetch tile it + NST - 1 into the buffer that tile it - 1 has left
    if (it + NST - 1 < n_tiles) load_tile((it + NST - 1) % NST, tile_lo + it + NST - 1);
    cp_async_commit();
    const __nv_bfloat16* kt = k_s + buf * BN * LD;
    const __nv_bfloat16* vt = v_s + buf * BN * LD;

    // ---- S = Q K^T ------------------------------------------------------------------
    float s[ST][4];
#pragma unroll
    for (int j = 0; j < ST; ++j) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.f;
#pragma unroll
    for (int ks = 0; ks < QSTEPS; ++ks) {
      if (SIZED && ks * 16 >= wcols) continue;
#pragma unroll
      for (int j = 0; j < ST; j += 2) {
        unsigned kb[4];
        const int key = wkey + j * 8 + (lane & 7) + (lane >> 4) * 8;
        const int dim = wcol + ks * 16 + ((lane >> 3) & 1) * 8;
        ldmatrix_x4(kb, kt + key * LD + dim);
        mma_bf16(s[j], qf[ks], kb[0], kb[1]);
        mma_bf16(s[j + 1], qf[ks], kb[2], kb[3]);
      }
    }
    // ---- mask, online softmax (exp2 domain) -----------------------------------------
    float m_new[2] = {m_run[0], m_run[1]};
    // A tile strictly inside every row's visible range needs no mask (the common case in decode).
    const bool inner = pooled ? key0 + BN <= nb_first && row0 + PB <= n_rows
                              : key0 + BN - 1 <= pos_first && key0 >= lo_last && row0 + PB <= n_rows &&
                                    !(GEN && p.slopes) && !(EXT && p.rel);
    if (inner) {
#pragma unroll
      for (int j = 0; j < ST; ++j) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          s[j][e] = score_log2<GEN>(p, s[j][e]);
          m_new[e >> 1] = fmaxf(m_new[e >> 1], s[j][e]);
        }
      }
    } else {
#pragma unroll
      for (int j = 0; j < ST; ++j) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int i = e >> 1;
          const int key = key0 + wkey + j * 8 + tig * 2 + (e & 1);
          bool vis = row_ok[i] && key <= row_pos[i] && key >= row_lo[i];
          float off = row_slope[i] * (float)(row_pos[i] - key);
          if (EXT) {
            if (pooled) {
              vis = key < row_blocks[i];
              off = 0.f;
            } else if (vis && p.rel) {
              const int at = min(row_pos[i] - key, p.rel_len - 1);
              off -= p.rel_staged ? rel_s[row_head[i] * p.rel_len + at] : row_rel[i][at] * 1.4426950408889634f;
            }
          }
          const float v = vis ? score_log2<GEN>(p, s[j][e], off) : -INFINITY;
          s[j][e] = v;
          m_new[i] = fmaxf(m_new[i], v);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      m_new[i] = fmaxf(m_new[i], __shfl_xor_sync(0xffffffffu, m_new[i], 1));
      m_new[i] = fmaxf(m_new[i], __shfl_xor_sync(0xffffffffu, m_new[i], 2));
    }
    float corr[2], base[2], l_add[2] = {0.f, 0.f};
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      base[i] = (m_new[i] == -INFINITY) ? 0.f : m_new[i];
      corr[i] = exp2f(m_run[i] - base[i]);          // m_run = -inf gives 0
      m_run[i] = m_new[i];
    }
    if constexpr (!GEN) {
      unsigned pf[ST / 2][4];
#pragma unroll
      for (int j = 0; j < ST; ++j) {
        const float p0 = exp2f(s[j][0] - base[0]), p1 = exp2f(s[j][1] - base[0]);
        const float p2 = exp2f(s[j][2] - base[1]), p3 = exp2f(s[j][3] - base[1]);
        l_add[0] += p0 + p1;
        l_add[1] += p2 + p3;
        pf[j >> 1][(j & 1) * 2 + 0] = pack_bf16(p0, p1);
        pf[j >> 1][(j & 1) * 2 + 1] = pack_bf16(p2, p3);
      }
#pragma unroll
      for (int i = 0; i < 2; ++i) l_run[i] = l_run[i] * corr[i] + l_add[i];
#pragma unroll
      for (int d = 0; d < DT; ++d) {
        o[d][0] *= corr[0]; o[d][1] *= corr[0];
        o[d][2] *= corr[1]; o[d][3] *= corr[1];
      }
      // ---- O += P V -------------------------------------------------------------------
#pragma unroll
      for (int kk = 0; kk < ST / 2; ++kk) {
#pragma unroll
        for (int d = 0; d < DT; d += 2) {
          if (SIZED && d * 8 >= vs) continue;
          unsigned vb[4];
          const int key = wkey + kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8;
          const int dim = d * 8 + (lane >> 4) * 8;
          ldmatrix_x4_trans(vb, vt + key * LD + dim);
          mma_bf16(o[d], pf[kk], vb[0], vb[1]);
          mma_bf16(o[d + 1], pf[kk], vb[2], vb[3]);
        }
      }
    } else {
      // The weights stay float32 in s[][]; each block of 16 keys is split into its bfloat16 rounding and the
      // bfloat16 rounding of what that left over right before it meets V, so no second copy of P is held.
#pragma unroll
      for (int j = 0; j < ST; ++j) {
        s[j][0] = exp2f(s[j][0] - base[0]); s[j][1] = exp2f(s[j][1] - base[0]);
        s[j][2] = exp2f(s[j][2] - base[1]); s[j][3] = exp2f(s[j][3] - base[1]);
        l_add[0] += s[j][0] + s[j][1];
        l_add[1] += s[j][2] + s[j][3];
      }
#pragma unroll
      for (int i = 0; i < 2; ++i) l_run[i] = l_run[i] * corr[i] + l_add[i];
#pragma unroll
      for (int d = 0; d < DT; ++d) {
        o[d][0] *= corr[0]; o[d][1] *= corr[0];
        o[d][2] *= corr[1]; o[d][3] *= corr[1];
      }
#pragma unroll
      for (int kk = 0; kk < ST / 2; ++kk) {
        unsigned hi[4], lo[4];
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const float* pv = s[2 * kk + half];
          float r[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) r[e] = pv[e] - __bfloat162float(__float2bfloat16_rn(pv[e]));
          hi[half * 2 + 0] = pack_bf16(pv[0], pv[1]);
          hi[half * 2 + 1] = pack_bf16(pv[2], pv[3]);
          lo[half * 2 + 0] = pack_bf16(r[0], r[1]);
          lo[half * 2 + 1] = pack_bf16(r[2], r[3]);
        }
#pragma unroll
        for (int d = 0; d < DT; d += 2) {
          if (SIZED && d * 8 >= vs) continue;
          unsigned vb[4];
          const int key = wkey + kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8;
          const int dim = d * 8 + (lane >> 4) * 8;
          ldmatrix_x4_trans(vb, vt + key * LD + dim);
          mma_bf16(o[d], hi, vb[0], vb[1]);
          mma_bf16(o[d + 1], hi, vb[2], vb[3]);
          mma_bf16(o[d], lo, vb[0], vb[1]);
          mma_bf16(o[d + 1], lo, vb[2], vb[3]);
        }
      }
    }
    cp_async_wait<NST - 2>();   // tile it + 1 has landed (later ones may still fly)
    __syncthreads();
  }

  // ---- finish -----------------------------------------------------------------------
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    l_run[i] += __shfl_xor_sync(0xffffffffu, l_run[i], 1);
    l_run[i] += __shfl_xor_sync(0xffffffffu, l_run[i], 2);
  }
  if constexpr (DEC) {
    // The four warps hold partial states of the same 16 rows: merge them in warp order.
    float* mo = reinterpret_cast<float*>(k_s);        // [NWARPS][16][HS]
    float* mml = reinterpret_cast<float*>(v_s);       // [NWARPS][16][2]
    __syncthreads();                                    // every warp is done with the K/V tiles
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int r = gid + i * 8;
#pragma unroll
      for (int d = 0; d < DT; ++d)
        *reinterpret_cast<float2*>(mo + ((size_t)warp * 16 + r) * HS + d * 8 + tig * 2) =
            make_float2(o[d][i * 2], o[d][i * 2 + 1]);
      if (tig == 0) {
        mml[(warp * 16 + r) * 2] = m_run[i];
        mml[(warp * 16 + r) * 2 + 1] = l_run[i];
      }
    }
    __syncthreads();
    if constexpr (MAPS) {
      float* os = mo + NWARPS * 16 * HS;              // [PB][vs]: the difference of the maps
      const int pairs = min(PB, n_rows - row0);
      // what the four warps have for a row and column: (maximum, sum of weights, weighted values)
      auto merged = [&](int r, int d) {
        float mm = -INFINITY, ll = 0.f, acc = 0.f;
#pragma unroll
        for (int w = 0; w < NWARPS; ++w) mm = fmaxf(mm, mml[(w * 16 + r) * 2]);
#pragma unroll
        for (int w = 0; w < NWARPS; ++w) {
          const float m = mml[(w * 16 + r) * 2];
          const float f = (m == -INFINITY) ? 0.f : exp2f(m - mm);
          ll += mml[(w * 16 + r) * 2 + 1] * f;
          acc += mo[((size_t)w * 16 + r) * HS + d] * f;
        }
        return make_float3(mm, ll, acc);
      };
      // the norm of every pair's difference and the store: a warp per pair
      auto store_pairs = [&]() {
        __syncthreads();
        for (int u = warp; u < pairs; u += NWARPS) {
          const int row = row0 + u, t = row / p.per, h = row - t * p.per;
          float ss = 0.f;
          for (int d = lane; d < vs; d += 32) ss = __fmaf_rn(os[u * vs + d], os[u * vs + d], ss);
          const float r = p.out_scale / sqrtf(warp_sum(ss) / (float)vs + p.diff_eps);
          __nv_bfloat16* dst = p.out + (size_t)(tok0 + t) * p.out_stride + (size_t)(kvh * p.per + h) * vs;
          for (int d = lane; d < vs; d += 32) dst[d] = __float2bfloat16_rn(os[u * vs + d] * r);
        }
      };
      if (p.n_splits == 1) {
        for (int e = threadIdx.x; e < pairs * vs; e += NWARPS * 32) {
          const int u = e / vs, d = e - u * vs;
          const float3 a = merged(u, d), b = merged(u + PB, d);
          os[e] = a.z / a.y - p.lambda * (b.z / b.y);
        }
        store_pairs();
        return;
      }
      for (int e = threadIdx.x; e < 2 * pairs * vs; e += NWARPS * 32) {
        const int ru = e / vs, d = e - ru * vs;
        const int map = ru >= pairs, u = ru - map * pairs;
        const int row = row0 + u, t = row / p.per, h = row - t * p.per;
        const size_t slot = (((size_t)(tok0 + t) * p.nh + kvh * p.per + h) * 2 + map) * p.n_splits + split;
        const float3 a = merged(u + map * PB, d);
        p.part_o[slot * vs + d] = a.z;
        if (d == 0) {
          p.part_ml[slot * 2] = a.x;
          p.part_ml[slot * 2 + 1] = a.y;
        }
      }
      __shared__ int s_done;
      int32_t* ticket = p.tickets + (size_t)blockIdx.y * gridDim.x + blockIdx.x;
      __threadfence();
      __syncthreads();
      if (threadIdx.x == 0) s_done = (atomicAdd(ticket, 1) == p.n_splits - 1) ? 1 : 0;
      __syncthreads();
      if (!s_done) return;
      __threadfence();
      for (int e = threadIdx.x; e < pairs * vs; e += NWARPS * 32) {
        const int u = e / vs, d = e - u * vs;
        const int row = row0 + u, t = row / p.per, h = row - t * p.per;
        const volatile float* ml = p.part_ml;
        const volatile float* po = p.part_o;
        float res[2];
#pragma unroll
        for (int map = 0; map < 2; ++map) {
          const size_t base = (((size_t)(tok0 + t) * p.nh + kvh * p.per + h) * 2 + map) * p.n_splits;
          float mm = -INFINITY, ll = 0.f, acc = 0.f;
          for (int sp = 0; sp < p.n_splits; ++sp) mm = fmaxf(mm, ml[(base + sp) * 2]);
          for (int sp = 0; sp < p.n_splits; ++sp) {
            const float m = ml[(base + sp) * 2];
            const float f = (m == -INFINITY) ? 0.f : exp2f(m - mm);
            ll += ml[(base + sp) * 2 + 1] * f;
            acc += po[(base + sp) * vs + d] * f;
          }
          res[map] = acc / ll;
        }
        os[e] = res[0] - p.lambda * res[1];
      }
      store_pairs();
      if (threadIdx.x == 0) *ticket = 0;
      return;
    }
    const int rows_here = min(16, n_rows - row0);
    for (int e = threadIdx.x; e < rows_here * vs; e += NWARPS * 32) {
      const int r = e / vs, d = e - r * vs;
      float mm = -INFINITY;
#pragma unroll
      for (int w = 0; w < NWARPS; ++w) mm = fmaxf(mm, mml[(w * 16 + r) * 2]);
      float ll = 0.f, acc = 0.f;
#pragma unroll
      for (int w = 0; w < NWARPS; ++w) {
        const float m = mml[(w * 16 + r) * 2];
        const float f = (m == -INFINITY) ? 0.f : exp2f(m - mm);
        ll += mml[(w * 16 + r) * 2 + 1] * f;
        acc += mo[((size_t)w * 16 + r) * HS + d] * f;
      }
      const int row = row0 + r;
      const int t = row / p.per, h = row - t * p.per;
      const int tok = tok0 + t, head = kvh * p.per + h;
      if (p.n_splits == 1) {
        float sz = 0.f;
        if (GEN && p.sink) {
          sz = sink_log2(p, head);
          const float up = fmaxf(mm, sz);           // the sink may be the row's largest score
          acc *= exp2f(mm - up);
          ll = ll * exp2f(mm - up);
          mm = up;
        }
        float res = acc * finish_factor<GEN>(p, mm, ll, sz);
        if (GEN && p.gate) res *= gate_factor(p, tok, head, vs, d);
        p.out[(size_t)tok * p.out_stride + (size_t)head * vs + d] = __float2bfloat16_rn(res);
      } else {
        const size_t slot = ((size_t)tok * p.nh + head) * p.n_splits + split;
        p.part_o[slot * vs + d] = acc;
        if (d == 0) {
          p.part_ml[slot * 2] = mm;
          p.part_ml[slot * 2 + 1] = ll;
        }
      }
    }
    if (p.n_splits > 1) {
      // Ticket: the block that finds every other split already done merges them all.
      __shared__ int s_last;
      __threadfence();
      __syncthreads();
      if (threadIdx.x == 0) s_last = (atomicAdd(&p.tickets[blockIdx.y], 1) == p.n_splits - 1) ? 1 : 0;
      __syncthreads();
      if (s_last) {
        __threadfence();
        for (int e = threadIdx.x; e < rows_here * vs; e += NWARPS * 32) {
          const int r = e / vs, d = e - r * vs;
          const int row = row0 + r;
          const int t = row / p.per, h = row - t * p.per;
          const int tok = tok0 + t, head = kvh * p.per + h;
          const size_t base = ((size_t)tok * p.nh + head) * p.n_splits;
          const volatile float* ml = p.part_ml;
          const volatile float* po = p.part_o;
          float mm = -INFINITY;
          for (int sp = 0; sp < p.n_splits; ++sp) mm = fmaxf(mm, ml[(base + sp) * 2]);
          float ll = 0.f, acc = 0.f;
          for (int sp = 0; sp < p.n_splits; ++sp) {
            const float m = ml[(base + sp) * 2];
            const float f = (m == -INFINITY) ? 0.f : exp2f(m - mm);
            ll += ml[(base + sp) * 2 + 1] * f;
            acc += po[(base + sp) * vs + d] * f;
          }
          float sz = 0.f;
          if (GEN && p.sink) {
            sz = sink_log2(p, head);
            const float up = fmaxf(mm, sz);
            acc *= exp2f(mm - up);
            ll = ll * exp2f(mm - up);
            mm = up;
          }
          float res = acc * finish_factor<GEN>(p, mm, ll, sz);
          if (GEN && p.gate) res *= gate_factor(p, tok, head, vs, d);
          p.out[(size_t)tok * p.out_stride + (size_t)head * vs + d] = __float2bfloat16_rn(res);
        }
        if (threadIdx.x == 0) p.tickets[blockIdx.y] = 0;
      }
    }
  } else if constexpr (MAPS) {
    // The second map's warps leave their results in shared memory; the first map's warps take lambda times them off.
    constexpr int OLD = HS + 8;
    float* other = reinterpret_cast<float*>(k_s);     // [PB][OLD] (fits the two K tiles)
    static_assert(PB * OLD * sizeof(float) <= NST * BN * LD * sizeof(__nv_bfloat16), "the second map's results must fit");
    __syncthreads();                                  // every warp is done with the K tiles
    if (wrow >= PB) {
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const float inv = l_run[i] > 0.f ? 1.0f / l_run[i] : 0.f;
        float* dst = other + (wrow - PB + gid + i * 8) * OLD;
#pragma unroll
        for (int d = 0; d < DT; ++d)
          if (d * 8 < vs) *reinterpret_cast<float2*>(dst + d * 8 + tig * 2) = make_float2(o[d][i * 2] * inv, o[d][i * 2 + 1] * inv);
      }
    }
    __syncthreads();
    if (wrow >= PB) return;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const float inv = l_run[i] > 0.f ? 1.0f / l_run[i] : 0.f;
      const float* src = other + (wrow + gid + i * 8) * OLD;
      float ss = 0.f;
#pragma unroll
      for (int d = 0; d < DT; ++d) {
        if (d * 8 >= vs) continue;
        const float2 b = *reinterpret_cast<const float2*>(src + d * 8 + tig * 2);
        o[d][i * 2] = o[d][i * 2] * inv - p.lambda * b.x;
        o[d][i * 2 + 1] = o[d][i * 2 + 1] * inv - p.lambda * b.y;
        ss = __fmaf_rn(o[d][i * 2], o[d][i * 2], ss);
        ss = __fmaf_rn(o[d][i * 2 + 1], o[d][i * 2 + 1], ss);
      }
      ss += __shfl_xor_sync(0xffffffffu, ss, 1);      // the four lanes of a row
      ss += __shfl_xor_sync(0xffffffffu, ss, 2);
      if (!row_ok[i]) continue;
      const float r = p.out_scale / sqrtf(ss / (float)vs + p.diff_eps);
      const int row = row0 + wrow + gid + i * 8;
      const int t = row / p.per, h = row - t * p.per;
      __nv_bfloat16* dst = p.out + (size_t)(tok0 + t) * p.out_stride + (size_t)(kvh * p.per + h) * vs;
#pragma unroll
      for (int d = 0; d < DT; ++d)
        if (d * 8 < vs)
          *reinterpret_cast<__nv_bfloat162*>(dst + d * 8 + tig * 2) = __floats2bfloat162_rn(o[d][i * 2] * r, o[d][i * 2 + 1] * r);
    }
  } else {
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    if (!row_ok[i]) continue;
    const int row = row0 + wrow + gid + i * 8;
    const int t = row / p.per, h = row - t * p.per;
    const int tok = tok0 + t, head = kvh * p.per + h;
    float inv;
    if (GEN && p.sink) {
      const float sz = sink_log2(p, head);
      const float up = fmaxf(m_run[i], sz);
      const float down = exp2f(m_run[i] - up);       // m_run = -inf (no visible key) gives 0
      inv = down * finish_factor<GEN>(p, up, l_run[i] * down, sz);
    } else {
      inv = finish_factor<GEN>(p, m_run[i], l_run[i]);
    }
    __nv_bfloat16* dst = p.out + (size_t)tok * p.out_stride + (size_t)head * vs;
#pragma unroll
    for (int d = 0; d < DT; ++d) {
      if (SIZED && d * 8 >= vs) continue;
      float v0 = o[d][i * 2] * inv, v1 = o[d][i * 2 + 1] * inv;
      if (GEN && p.gate) {
        v0 *= gate_factor(p, tok, head, vs, d * 8 + tig * 2);
        v1 *= gate_factor(p, tok, head, vs, d * 8 + tig * 2 + 1);
      }
      *reinterpret_cast<__nv_bfloat162*>(dst + d * 8 + tig * 2) = __floats2bfloat162_rn(v0, v1);
    }
  }
  }
}

template <int HS, bool DEC, int FORM>
int launch_mode(const AttnParams& args, int n_requests, int max_rows, cudaStream_t stream) {
  constexpr int LD = HS + 8;
  constexpr int RB = DEC ? 16 : BM, PB = FORM >= 4 ? RB / 2 : RB, NST = DEC ? 3 : 2;
  constexpr size_t tiles = (size_t)(RB + 2 * NST * BN) * LD * sizeof(__nv_bfloat16);
  // what a staged table of biases may take without costing a resident block
  constexpr int rel_room = FORM == 2 || FORM == 3 ? (DEC ? 1024 : 4096) : 0;
  AttnParams p = args;
  p.rel_staged = p.rel != nullptr && p.per * p.rel_len <= rel_room;
  const size_t smem = tiles + (p.rel_staged ? (size_t)p.per * p.rel_len * sizeof(float) : 0);
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(paged_attention_mma_kernel<HS, DEC, FORM>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                             (int)(tiles + rel_room * sizeof(float))) != cudaSuccess)
      return YALIS_ERR_LAUNCH;
    configured = true;
  }
  dim3 grid((max_rows + PB - 1) / PB, n_requests * p.g, p.n_splits);
  if (grid.y > 65535 || grid.z > 65535) return YALIS_ERR_SHAPE;
  return yalis_launch(paged_attention_mma_kernel<HS, DEC, FORM>, grid, dim3(NWARPS * 32), smem, stream, p);
}

template <int HS>
int launch(const AttnParams& p, int n_requests, int max_rows, cudaStream_t stream) {
  const bool general = p.cap_log2 > 0.f || p.sink || p.out_scale != 1.0f || p.exact_weights || p.chunk > 0 || p.slopes || p.gate;
  if (general)
    return max_rows <= 16 ? launch_mode<HS, true, 1>(p, n_requests, max_rows, stream)
                          : launch_mode<HS, false, 1>(p, n_requests, max_rows, stream);
  return max_rows <= 16 ? launch_mode<HS, true, 0>(p, n_requests, max_rows, stream)
                        : launch_mode<HS, false, 0>(p, n_requests, max_rows, stream);
}

template <int HS>
int launch_extended(const AttnParams& p, int n_requests, int max_rows, cudaStream_t stream) {
  if (p.hs == HS && p.vs == HS)
    return max_rows <= 16 ? launch_mode<HS, true, 2>(p, n_requests, max_rows, stream)
                          : launch_mode<HS, false, 2>(p, n_requests, max_rows, stream);
  return max_rows <= 16 ? launch_mode<HS, true, 3>(p, n_requests, max_rows, stream)
                        : launch_mode<HS, false, 3>(p, n_requests, max_rows, stream);
}

template <int HS>
int launch_maps(const AttnParams& p, int n_requests, int max_pairs, cudaStream_t stream) {
  if (p.hs == HS && p.vs == HS)
    return max_pairs <= 16 ? launch_mode<HS, true, 5>(p, n_requests, max_pairs, stream)
                           : launch_mode<HS, false, 5>(p, n_requests, max_pairs, stream);
  return max_pairs <= 16 ? launch_mode<HS, true, 4>(p, n_requests, max_pairs, stream)
                         : launch_mode<HS, false, 4>(p, n_requests, max_pairs, stream);
}

}  // namespace

// Head sizes this kernel is built for.
YALIS_API int yalis_attention_mma_supports(int hs) {
  switch (hs) {
    case 16: case 32: case 48: case 64: case 80: case 96: case 112: case 128: case 160: case 192: case 224: case 256:
      return 1;
    default:
      return 0;
  }
}

// Whether the extended form takes keys of size hs and values of size vs.
YALIS_API int yalis_attention_mma_extended_supports(int hs, int vs) {
  return hs >= 8 && vs >= 8 && hs <= 256 && vs <= 256 && hs % 8 == 0 && vs % 8 == 0;
}

// Whether the form of two maps takes queries and keys of size d per map and values of size vs.
YALIS_API int yalis_attention_mma_maps_supports(int d, int vs) {
  return d >= 16 && d <= 128 && d % 16 == 0 && vs >= 8 && vs <= 256 && vs % 8 == 0;
}

// Scratch floats (hs: the size of a value) needed for n_splits > 1: part_o then part_ml.  Besides, `tickets` needs
// n_requests * g int32 that are zero before the first launch (each launch leaves them zero).
YALIS_API long long yalis_attention_mma_scratch_floats(int n_tokens, int nh, int hs, int n_splits) {
  return n_splits > 1 ? (long long)n_tokens * nh * n_splits * (hs + 2) : 0;
}

// softcap 0: none.  With a cap, a sink, a factor other than 1 or exact_weights the general form of the kernel runs;
// with vs != hs, a bias per distance (rel), pooled blocks (pool > 0) or a head size that has no kernel of its own the
// extended form.  maps 2: the form of two maps, hs the size of both maps' keys together and nh heads of two queries each
// (no soft cap, sink, chunk, slopes, gate, rel or pooled blocks); a step may be split while its pairs (token, head) of a
// request and key/value head are at most 16, with two partial results per head and a ticket per 8 pairs.
YALIS_API int yalis_paged_attention_mma_general(const void* q, int q_stride, void* out, int out_stride, const void* k_pool,
                                                const void* v_pool, const int32_t* positions, const int32_t* q_start,
                                                const int32_t* req_of_token, const int32_t* block_table, int table_width,
                                                int page_size, int num_pages, int n_tokens, int n_requests, int max_q_len,
                                                int nh, int g, int hs, float scale, int window, int n_splits, float* scratch,
                                                int32_t* tickets, float softcap, int sink, float out_scale,
                                                int exact_weights, int chunk, const float* sink_logits,
                                                const float* slopes, const void* gate, int gate_stride,
                                                int gate_per_head, int vs, const float* rel, int rel_len, int pool,
                                                const void* pk_pool, const void* pv_pool, const int32_t* pool_table,
                                                int pool_table_width, int pool_page_size, int pool_num_pages, int maps,
                                                float lambda, float diff_eps, cudaStream_t stream) {
  if (n_tokens <= 0 || n_requests <= 0) return YALIS_OK;
  if (softcap < 0.f) return YALIS_ERR_SHAPE;
  if (maps != 1 && (maps != 2 || hs % 2 || !yalis_attention_mma_maps_supports(hs / 2, vs) || softcap > 0.f || sink || chunk > 0 ||
                    slopes || gate || rel || pool > 0))
    return YALIS_ERR_SHAPE;
  if (g <= 0 || nh % g != 0 || n_splits < 1 || max_q_len < 1) return YALIS_ERR_SHAPE;
  if (((uintptr_t)q | (uintptr_t)k_pool | (uintptr_t)v_pool | (uintptr_t)out) & 15) return YALIS_ERR_ALIGN;
  if ((q_stride % 8) || (out_stride % 2)) return YALIS_ERR_ALIGN;
  AttnParams p;
  p.q = (const __nv_bfloat16*)q; p.q_stride = q_stride;
  p.out = (__nv_bfloat16*)out; p.out_stride = out_stride;
  p.k_pool = (const __nv_bfloat16*)k_pool; p.v_pool = (const __nv_bfloat16*)v_pool;
  p.positions = positions; p.q_start = q_start; p.block_table = block_table;
  p.table_width = table_width; p.page_size = page_size; p.num_pages = num_pages;
  p.page_shift = -1;
  for (int sh = 0; sh < 31; ++sh)
    if ((1 << sh) == page_size) p.page_shift = sh;
  p.nh = nh; p.g = g; p.per = nh / g;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.cap_log2 = softcap * 1.4426950408889634f;
  p.scale_over_cap = softcap > 0.f ? scale / softcap : 0.f;
  p.sink = sink; p.out_scale = out_scale; p.exact_weights = exact_weights;
  p.window = window; p.n_splits = n_splits;
  p.chunk = chunk; p.sink_logits = sink ? sink_logits : nullptr; p.slopes = slopes;
  p.gate = (const __nv_bfloat16*)gate; p.gate_stride = gate_stride; p.gate_per_head = gate_per_head;
  p.hs = hs; p.vs = vs; p.rel = rel; p.rel_len = rel_len; p.pool = pool;
  p.pk_pool = (const __nv_bfloat16*)pk_pool; p.pv_pool = (const __nv_bfloat16*)pv_pool; p.pool_table = pool_table;
  p.pool_table_width = pool_table_width; p.pool_page_size = pool_page_size; p.pool_num_pages = pool_num_pages;
  p.pool_page_shift = -1;
  for (int sh = 0; sh < 31; ++sh)
    if ((1 << sh) == pool_page_size) p.pool_page_shift = sh;
  p.map_dim = hs / 2; p.lambda = lambda; p.diff_eps = diff_eps;
  const bool extended = vs != hs || rel != nullptr || pool > 0 || !yalis_attention_mma_supports(hs);
  if (pool < 0 || (rel && rel_len < 1)) return YALIS_ERR_SHAPE;
  if (pool > 0) {
    if (window <= 0 || chunk > 0 || !pk_pool || !pv_pool || !pool_table || pool_page_size < 1) return YALIS_ERR_SHAPE;
    if (((uintptr_t)pk_pool | (uintptr_t)pv_pool) & 15) return YALIS_ERR_ALIGN;
  }
  if (extended && !yalis_attention_mma_extended_supports(hs, vs)) return YALIS_ERR_SHAPE;
  if (chunk < 0) return YALIS_ERR_SHAPE;
  p.part_o = nullptr; p.part_ml = nullptr; p.tickets = tickets;
  if (n_splits > 1) {
    if (scratch == nullptr || tickets == nullptr || max_q_len * p.per > 16) return YALIS_ERR_SHAPE;
    p.part_o = scratch;
    p.part_ml = scratch + (size_t)n_tokens * nh * maps * n_splits * vs;
  }
  const int max_rows = max_q_len * p.per;
  int st;
  if (maps == 2) {
    const int widest = hs > vs ? hs : vs;
    if (widest <= 64) return launch_maps<64>(p, n_requests, max_rows, stream);
    if (widest <= 128) return launch_maps<128>(p, n_requests, max_rows, stream);
    return launch_maps<256>(p, n_requests, max_rows, stream);
  }
  if (extended) {
    const int widest = hs > vs ? hs : vs;
    if (widest <= 64) return launch_extended<64>(p, n_requests, max_rows, stream);
    if (widest <= 128) return launch_extended<128>(p, n_requests, max_rows, stream);
    return launch_extended<256>(p, n_requests, max_rows, stream);
  }
  switch (hs) {
    case 16: st = launch<16>(p, n_requests, max_rows, stream); break;
    case 32: st = launch<32>(p, n_requests, max_rows, stream); break;
    case 48: st = launch<48>(p, n_requests, max_rows, stream); break;
    case 64: st = launch<64>(p, n_requests, max_rows, stream); break;
    case 80: st = launch<80>(p, n_requests, max_rows, stream); break;
    case 96: st = launch<96>(p, n_requests, max_rows, stream); break;
    case 112: st = launch<112>(p, n_requests, max_rows, stream); break;
    case 128: st = launch<128>(p, n_requests, max_rows, stream); break;
    case 160: st = launch<160>(p, n_requests, max_rows, stream); break;
    case 192: st = launch<192>(p, n_requests, max_rows, stream); break;
    case 224: st = launch<224>(p, n_requests, max_rows, stream); break;
    case 256: st = launch<256>(p, n_requests, max_rows, stream); break;
    default: return YALIS_ERR_SHAPE;
  }
  return st;
}

// ---------------------------------------------------------------------------------------
// The same kernel with its temporary memory in a fixed array of the library, for callers that
// must not allocate (see attention_noalloc.h for who they are and for the rules).
// ---------------------------------------------------------------------------------------
#include <atomic>

#include "attention_noalloc.h"

namespace {

// Counters first (must be zero when a launch starts), then the partial results.  The name is
// usable as an address in device code only; host code has to ask the runtime for its address.
static __device__ __align__(256) unsigned char g_noalloc_scratch[YALIS_NOALLOC_SCRATCH_BYTES];

constexpr int kMaxDevices = 64;
// Device address of the array, per device.  Threads that make a device's first call at the same time all ask
// the runtime and store the same address: the slots are atomic so that none of them reads a half-written one.
std::atomic<void*> g_noalloc_ptr[kMaxDevices];

// Device address of the array on the current device; looked up on the first call there.
int noalloc_scratch(unsigned char** ptr) {
  int dev = -1;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= kMaxDevices) return YALIS_ERR_LAUNCH;
  void* p = g_noalloc_ptr[dev].load(std::memory_order_acquire);
  if (p == nullptr) {
    if (cudaGetSymbolAddress(&p, g_noalloc_scratch) != cudaSuccess || p == nullptr) return YALIS_ERR_LAUNCH;
    g_noalloc_ptr[dev].store(p, std::memory_order_release);
  }
  *ptr = static_cast<unsigned char*>(p);
  return YALIS_OK;
}

}  // namespace

YALIS_API int yalis_paged_attention_mma(const void* q, int q_stride, void* out, int out_stride, const void* k_pool,
                                        const void* v_pool, const int32_t* positions, const int32_t* q_start,
                                        const int32_t* req_of_token, const int32_t* block_table, int table_width,
                                        int page_size, int num_pages, int n_tokens, int n_requests, int max_q_len,
                                        int nh, int g, int hs, float scale, int window, int n_splits, float* scratch,
                                        int32_t* tickets, cudaStream_t stream) {
  return yalis_paged_attention_mma_general(q, q_stride, out, out_stride, k_pool, v_pool, positions, q_start, req_of_token,
                                           block_table, table_width, page_size, num_pages, n_tokens, n_requests, max_q_len,
                                           nh, g, hs, scale, window, n_splits, scratch, tickets, 0.f, 0, 1.0f, 0, 0, nullptr, nullptr,
                                           nullptr, 0, 0, hs, nullptr, 0, 0, nullptr, nullptr, nullptr, 0, 0, 0, 1, 0.f, 0.f, stream);
}

YALIS_API long long yalis_paged_attention_mma_noalloc_needed(int n_tokens, int n_requests, int nh, int g, int hs,
                                                             int n_splits, long long* ticket_bytes,
                                                             long long* partial_bytes) {
  const long long t = n_splits > 1 ? (long long)n_requests * g * (long long)sizeof(int32_t) : 0;
  const long long f = yalis_attention_mma_scratch_floats(n_tokens, nh, hs, n_splits) * (long long)sizeof(float);
  if (ticket_bytes) *ticket_bytes = t;
  if (partial_bytes) *partial_bytes = f;
  return t + f;
}

YALIS_API int yalis_paged_attention_mma_noalloc(const void* q, int q_stride, void* out, int out_stride,
                                                const void* k_pool, const void* v_pool, const int32_t* positions,
                                                const int32_t* q_start, const int32_t* req_of_token,
                                                const int32_t* block_table, int table_width, int page_size,
                                                int num_pages, int n_tokens, int n_requests, int max_q_len, int nh,
                                                int g, int hs, float scale, int window, int n_splits,
                                                cudaStream_t stream) {
  if (n_tokens <= 0 || n_requests <= 0) return YALIS_OK;
  if (n_splits < 1 || g <= 0) return YALIS_ERR_SHAPE;
  long long ticket_bytes = 0, partial_bytes = 0;
  yalis_paged_attention_mma_noalloc_needed(n_tokens, n_requests, nh, g, hs, n_splits, &ticket_bytes, &partial_bytes);
  if (ticket_bytes > YALIS_NOALLOC_TICKET_BYTES || partial_bytes > YALIS_NOALLOC_PARTIAL_BYTES)
    return YALIS_ERR_SCRATCH;                       // refused: nothing was launched
  unsigned char* base = nullptr;
  if (int st = noalloc_scratch(&base)) return st;
  int32_t* tickets = reinterpret_cast<int32_t*>(base);
  float* partials = reinterpret_cast<float*>(base + YALIS_NOALLOC_TICKET_BYTES);
  if (n_splits > 1) {
    // The array keeps what the last call left: the counters have to start at zero.
    if (cudaMemsetAsync(tickets, 0, (size_t)ticket_bytes, stream) != cudaSuccess) return YALIS_ERR_LAUNCH;
  }
  return yalis_paged_attention_mma(q, q_stride, out, out_stride, k_pool, v_pool, positions, q_start, req_of_token,
                                   block_table, table_width, page_size, num_pages, n_tokens, n_requests, max_q_len, nh,
                                   g, hs, scale, window, n_splits, n_splits > 1 ? partials : nullptr,
                                   n_splits > 1 ? tickets : nullptr, stream);
}
