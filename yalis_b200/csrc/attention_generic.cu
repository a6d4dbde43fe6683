// Paged causal attention, the exact one: any head size up to 256 (even), any
// number of heads and KV groups, any page size, float32 or bfloat16 storage,
// float32 arithmetic throughout.  One block per (token, head); each warp walks
// every fourth visible key in ascending order with an online softmax and the
// four partial results are merged in warp order.  For a given (position, head)
// the order of every sum is therefore fixed, whatever else is in the batch and
// however the request was cut into steps.  It is the kernel of the float32
// path and the twin against which the faster bfloat16 kernels are tested.
//
//   S = (q . k_j) * scale for keys j with  pos - window < j <= pos   (window 0: all j <= pos)
//   with chunk C > 0 also  j >= floor(pos / C) * C      (position 0 starts the first chunk)
//   S <- S - slope_h * (pos - j)                                        (slopes given only)
//   S <- cap * tanh(S / cap)                                            (cap > 0 only)
//   O = softmax(S) V, or with a sink: exp(S_j) / (exp(z_h) + sum_i exp(S_i)) V  (a key of score z_h and no value;
//   z_h = sink_logits[h], or 0 without that array)
//   O <- O * sigmoid(gate[t, h, :]), or * sigmoid(gate[t, h])           (gate given only)
//   S <- S + rel[h][min(pos - j, rel_len - 1)]                          (a bias per distance, given only)
// Pooled blocks (pool P > 0, with a window): beside the keys of the window a position sees one key and value for every
// block of P positions that lies wholly before it, blocks b < floor((pos - window + 1) / P); they come from pools of
// their own (entry b of the request's block table over entries) and share the softmax with the window's keys.
// Values may have a head size of their own (hsv).
// Two maps (maps = 2): a query head has two queries and a key/value head two keys per position (each of size hs, side by
// side in the query matrix and in a cached row of 2 hs), and one value; each map is a softmax of its own over the visible
// keys.  With O1, O2 the maps' results  O = O1 - lambda * O2,  O <- O / sqrt(mean(O^2) + eps) * out_scale.
// Mask by absolute position: yalis/attention/backend_impl/sdpa_and_flex.py:15-19, 301-307.
// KV head of query head h: h / (nh / g)                                 (:59-67).
#include "common.cuh"

namespace {

constexpr int kWarps = 4;
constexpr int kMaxPerLane = 8;  // head size <= 256

template <typename T>
struct GenericParams {
  const T* q; int q_stride;
  T* out; int out_stride;
  const T* k_pool; const T* v_pool;
  const int32_t* positions; const int32_t* req_of_token; const int32_t* block_table;
  int table_width, page_size, num_pages, nh, g, hs, hsv;
  float scale; int window; float softcap; int sink; float out_scale; int chunk;
  const float* sink_logits; const float* slopes;
  const float* rel; int rel_len;                 // [nh, rel_len] or null
  const T* gate; int gate_stride, gate_per_head; // [N, nh * hsv], or [N, nh] per head
  int pool;                                      // P > 0: pooled blocks before the window
  const T* pk_pool; const T* pv_pool; const int32_t* pool_table;
  int pool_table_width, pool_page_size, pool_num_pages;   // in entries (one per block)
  float lambda, diff_eps;                        // two maps
};

template <typename T, int MAPS>
__global__ void paged_attention_generic_kernel(const GenericParams<T> p) {
  extern __shared__ float smem[];  // per map [kWarps][hsv] accumulators, then m[kWarps], l[kWarps]; two maps: [hsv] besides
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, h = blockIdx.y;
  const int req = p.req_of_token[t];
  if (req < 0) return;
  const int pos = p.positions[t];
  const int kvh = h / (p.nh / p.g);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int per_lane = (p.hs + 31) >> 5, per_lane_v = (p.hsv + 31) >> 5;

  float qr[MAPS][kMaxPerLane], acc[MAPS][kMaxPerLane];
  const T* qp = p.q + (size_t)t * p.q_stride + (size_t)h * (MAPS * p.hs);
#pragma unroll
  for (int a = 0; a < MAPS; ++a)
#pragma unroll
    for (int i = 0; i < kMaxPerLane; ++i) {
      const int d = lane + 32 * i;
      qr[a][i] = (i < per_lane && d < p.hs) ? to_f32<T>(qp[a * p.hs + d]) : 0.f;
      acc[a][i] = 0.f;
    }
  float m[MAPS], l[MAPS];
#pragma unroll
  for (int a = 0; a < MAPS; ++a) {
    m[a] = -INFINITY;
    l[a] = 0.f;
  }
  int lo = (p.window > 0 && pos - p.window + 1 > 0) ? pos - p.window + 1 : 0;
  if (p.chunk > 0) lo = max(lo, (pos / p.chunk) * p.chunk);
  const float slope = p.slopes ? p.slopes[h] : 0.f;
  const int32_t* bt = p.block_table + (size_t)req * p.table_width;
  // the pooled blocks first, then the window's keys: one row of places, of which each warp walks every fourth
  const int blocks = (p.pool > 0 && p.window > 0 && pos - p.window + 1 > 0) ? (pos - p.window + 1) / p.pool : 0;
  for (int at = warp; at < blocks + pos - lo + 1; at += kWarps) {
    const bool pooled = at < blocks;
    const int j = pooled ? at : lo + (at - blocks);
    const int ps = pooled ? p.pool_page_size : p.page_size;
    const int pi = j / ps;
    const int32_t* table = pooled ? p.pool_table + (size_t)req * p.pool_table_width : bt;
    const int page = pi < (pooled ? p.pool_table_width : p.table_width) ? table[pi] : -1;
    if (page < 0 || page >= (pooled ? p.pool_num_pages : p.num_pages)) continue;  // unmapped: treated as masked
    const size_t row = ((size_t)page * p.g + kvh) * ps + (j - pi * ps);
    const T* kp = (pooled ? p.pk_pool : p.k_pool) + row * (MAPS * p.hs);
    const T* vp = (pooled ? p.pv_pool : p.v_pool) + row * p.hsv;
#pragma unroll
    for (int a = 0; a < MAPS; ++a) {
      float dot = 0.f;
#pragma unroll
      for (int i = 0; i < kMaxPerLane; ++i) {
        const int d = lane + 32 * i;
        if (i < per_lane && d < p.hs) dot += qr[a][i] * to_f32<T>(kp[a * p.hs + d]);
      }
      float s = warp_sum(dot) * p.scale;
      if (p.slopes && !pooled) s -= slope * (float)(pos - j);
      if (p.rel && !pooled) s += p.rel[(size_t)h * p.rel_len + min(pos - j, p.rel_len - 1)];
      if (p.softcap > 0.f) s = p.softcap * tanhf(s / p.softcap);
      const float m_new = fmaxf(m[a], s);
      const float corr = expf(m[a] - m_new);
      const float e = expf(s - m_new);
      l[a] = l[a] * corr + e;
#pragma unroll
      for (int i = 0; i < kMaxPerLane; ++i) {
        const int d = lane + 32 * i;
        if (i < per_lane_v && d < p.hsv) acc[a][i] = acc[a][i] * corr + e * to_f32<T>(vp[d]);
      }
      m[a] = m_new;
    }
  }
  const int map_floats = kWarps * p.hsv + 2 * kWarps;
#pragma unroll
  for (int a = 0; a < MAPS; ++a) {
    float* acc_w = smem + a * map_floats + warp * p.hsv;
#pragma unroll
    for (int i = 0; i < kMaxPerLane; ++i) {
      const int d = lane + 32 * i;
      if (i < per_lane_v && d < p.hsv) acc_w[d] = acc[a][i];
    }
    if (lane == 0) {
      smem[a * map_floats + kWarps * p.hsv + warp] = m[a];
      smem[a * map_floats + kWarps * p.hsv + kWarps + warp] = l[a];
    }
  }
  __syncthreads();
  if constexpr (MAPS == 2) {
    __shared__ float scratch[32];
    float* o_s = smem + 2 * map_floats;
    float wgt[2][kWarps];
#pragma unroll
    for (int a = 0; a < 2; ++a) {
      const float* ms = smem + a * map_floats + kWarps * p.hsv;
      const float* ls = ms + kWarps;
      float mm = -INFINITY, ll = 0.f;
#pragma unroll
      for (int w = 0; w < kWarps; ++w) mm = fmaxf(mm, ms[w]);
#pragma unroll
      for (int w = 0; w < kWarps; ++w) {
        wgt[a][w] = ms[w] == -INFINITY ? 0.f : expf(ms[w] - mm);
        ll += ls[w] * wgt[a][w];
      }
#pragma unroll
      for (int w = 0; w < kWarps; ++w) wgt[a][w] = ll > 0.f ? wgt[a][w] / ll : 0.f;
    }
    float ss = 0.f;
    for (int d = threadIdx.x; d < p.hsv; d += blockDim.x) {
      float o[2] = {0.f, 0.f};
#pragma unroll
      for (int a = 0; a < 2; ++a)
#pragma unroll
        for (int w = 0; w < kWarps; ++w) o[a] += smem[a * map_floats + w * p.hsv + d] * wgt[a][w];
      const float v = o[0] - p.lambda * o[1];
      o_s[d] = v;
      ss = __fmaf_rn(v, v, ss);
    }
    const float r = p.out_scale / sqrtf(block_sum(ss, scratch) / (float)p.hsv + p.diff_eps);
    T* op = p.out + (size_t)t * p.out_stride + (size_t)h * p.hsv;
    for (int d = threadIdx.x; d < p.hsv; d += blockDim.x) op[d] = from_f32<T>(o_s[d] * r);
    return;
  }
  const float* acc_s = smem;
  const float* m_s = smem + kWarps * p.hsv;
  const float* l_s = m_s + kWarps;
  float mm = -INFINITY;
#pragma unroll
  for (int w = 0; w < kWarps; ++w) mm = fmaxf(mm, m_s[w]);
  const float sink_z = (p.sink && p.sink_logits) ? p.sink_logits[h] : 0.f;
  if (p.sink) mm = fmaxf(mm, sink_z);
  float ll = p.sink ? expf(sink_z - mm) : 0.f;
  float wgt[kWarps];
#pragma unroll
  for (int w = 0; w < kWarps; ++w) {
    wgt[w] = (m_s[w] == -INFINITY) ? 0.f : expf(m_s[w] - mm);
    ll += l_s[w] * wgt[w];
  }
  T* op = p.out + (size_t)t * p.out_stride + (size_t)h * p.hsv;
  for (int d = threadIdx.x; d < p.hsv; d += blockDim.x) {
    float o = 0.f;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) o += acc_s[w * p.hsv + d] * wgt[w];
    float res = ll > 0.f ? o / ll * p.out_scale : 0.f;
    if (p.gate) {
      const size_t at = (size_t)t * p.gate_stride + (p.gate_per_head ? (size_t)h : (size_t)h * p.hsv + d);
      res *= 1.0f / (1.0f + expf(-to_f32<T>(p.gate[at])));
    }
    op[d] = from_f32<T>(res);
  }
}

}  // namespace

// maps 2: two maps, hs the size of one map's queries and keys; no sink, gate or pooled blocks.
// rel null: no bias per distance.  pool 0: no pooled blocks (the pool_* arguments are not read).
YALIS_API int yalis_paged_attention_generic(const void* q, int q_stride, void* out, int out_stride,
                                            const void* k_pool, const void* v_pool, int dtype,
                                            const int32_t* positions, const int32_t* req_of_token,
                                            const int32_t* block_table, int table_width, int page_size,
                                            int num_pages, int n_tokens, int nh, int g, int hs, int hsv,
                                            float scale, int window, float softcap, int sink, float out_scale,
                                            int chunk, const float* sink_logits, const float* slopes, const void* gate,
                                            int gate_stride, int gate_per_head, const float* rel, int rel_len, int pool,
                                            const void* pk_pool, const void* pv_pool, const int32_t* pool_table,
                                            int pool_table_width, int pool_page_size, int pool_num_pages, int maps,
                                            float lambda, float diff_eps, cudaStream_t stream) {
  if (n_tokens <= 0) return YALIS_OK;
  if (maps != 1 && (maps != 2 || sink || gate || pool > 0)) return YALIS_ERR_SHAPE;
  if (hs <= 0 || hs > 32 * kMaxPerLane || hsv <= 0 || hsv > 32 * kMaxPerLane || g <= 0 || nh % g != 0 || nh > 65535)
    return YALIS_ERR_SHAPE;
  if ((rel && rel_len < 1) || pool < 0 || (pool > 0 && (window <= 0 || chunk > 0 || !pk_pool || !pv_pool || !pool_table || pool_page_size < 1)))
    return YALIS_ERR_SHAPE;
  const size_t smem = (maps * ((size_t)kWarps * hsv + 2 * kWarps) + (maps == 2 ? hsv : 0)) * sizeof(float);
  dim3 grid(n_tokens, nh);
  YALIS_DISPATCH_DTYPE(dtype, T, {
    GenericParams<T> p;
    p.q = (const T*)q; p.q_stride = q_stride; p.out = (T*)out; p.out_stride = out_stride;
    p.k_pool = (const T*)k_pool; p.v_pool = (const T*)v_pool;
    p.positions = positions; p.req_of_token = req_of_token; p.block_table = block_table;
    p.table_width = table_width; p.page_size = page_size; p.num_pages = num_pages;
    p.nh = nh; p.g = g; p.hs = hs; p.hsv = hsv;
    p.scale = scale; p.window = window; p.softcap = softcap; p.sink = sink; p.out_scale = out_scale; p.chunk = chunk;
    p.sink_logits = sink_logits; p.slopes = slopes; p.rel = rel; p.rel_len = rel_len;
    p.gate = (const T*)gate; p.gate_stride = gate_stride; p.gate_per_head = gate_per_head;
    p.pool = pool; p.pk_pool = (const T*)pk_pool; p.pv_pool = (const T*)pv_pool; p.pool_table = pool_table;
    p.pool_table_width = pool_table_width; p.pool_page_size = pool_page_size; p.pool_num_pages = pool_num_pages;
    p.lambda = lambda; p.diff_eps = diff_eps;
    return maps == 2 ? yalis_launch(paged_attention_generic_kernel<T, 2>, grid, dim3(kWarps * 32), smem, stream, p)
                     : yalis_launch(paged_attention_generic_kernel<T, 1>, grid, dim3(kWarps * 32), smem, stream, p);
  });
  return YALIS_OK;
}
