// What lies between a mixer's input projection and its core, for mixers whose heads are
// prepared in more ways than a full rotation: an added bias, a norm over the head with a
// learned scale (or over all heads at once), a rotation of only the first `rot_dims` sizes, a
// constant factor, value heads of a size of their own.  Queries go to a plain matrix; keys and values go to the pages of a
// cache or to plain matrices (for mixers that keep a state instead of keys); blocks of P
// consecutive cached keys and values may be kept as their means besides.  Also the
// element-wise activations of dense feed-forwards and the row-wise additions of looped layers.
// All arithmetic is float32; sines and cosines come from sincosf of a float32 angle.
#include "common.cuh"

namespace {

constexpr int kMaxHeadDim = 1024;

struct PrepParams {
  const void* src; int src_stride;           // [N, ...]: q heads at q_off, k heads at k_off, v heads at v_off
  int q_off, k_off, v_off;
  const void* q_bias; const void* k_bias; const void* v_bias;     // model dtype, or null
  const float* q_norm; const float* k_norm; float norm_eps;       // scale over dim, or null: no norm
  const float* inv_freq; int rot_dims;                            // [rot_dims / 2], or null: no rotation
  int rot_interleaved;                                            // pair i is (2i, 2i + 1) instead of (i, i + rot_dims / 2)
  float rot_scale;                                                // factor on cosine and sine
  int norm_all;                                                   // the norm is over all heads of q (of k) at once, scales [heads * dim]
  float q_scale, k_scale;
  float q_temp_coef; int q_temp_every;                            // every > 0: q *= 1 + coef * ln(floor((pos + 1) / every) + 1)
  void* q_out; int q_out_stride;             // [N, nq * dim]
  void* k_out; int k_out_stride;             // plain destinations (used when k_pool is null)
  void* v_out; int v_out_stride;
  void* k_pool; void* v_pool;                // [pages, nk, page_size, dim] and [pages, nk, page_size, vdim]
  const int32_t* block_table; int table_width, page_size, num_pages;
  const int32_t* positions; const int32_t* req_of_token;
  int nq, nk, dim, vdim;
  int maps;                                  // keys per key/value head, side by side in its cached row [maps * dim] (1: the usual)
  int32_t* bad_page;
  int pool;                                  // P > 0: the warp that stores the last row of a block of P positions stores their mean
  void* pk_pool; void* pv_pool;              // [pages, nk, pool_page_size, dim] and [..., vdim], an entry per block
  const int32_t* pool_table; int pool_table_width, pool_page_size, pool_num_pages;
};

// Where a request's cached row `at` lies in pages of `page_size` rows: its index among the rows of one head, or -1.
__device__ __forceinline__ long long paged_row(const int32_t* table, int width, int page_size, int num_pages, int nk, int head,
                                               int at) {
  const int pi = at / page_size;
  const int page = pi < width ? table[pi] : -1;
  return page < 0 || page >= num_pages ? -1 : ((long long)page * nk + head) * page_size + (at - pi * page_size);
}

// The mean of a head's cached rows at positions pos - P + 1 .. pos, added in order in float32, goes to entry pos / P.
// One warp; every row must be stored and visible to it.
template <typename T>
__device__ void store_block_mean(const PrepParams& p, int req, int pos, int head, bool is_v, int lane) {
  const int width = is_v ? p.vdim : p.dim;
  const T* rows = reinterpret_cast<const T*>(is_v ? p.v_pool : p.k_pool);
  const int32_t* table = p.block_table + (size_t)req * p.table_width;
  const long long entry = paged_row(p.pool_table + (size_t)req * p.pool_table_width, p.pool_table_width, p.pool_page_size,
                                    p.pool_num_pages, p.nk, head, pos / p.pool);
  if (entry < 0) {
    if (lane == 0 && p.bad_page) atomicOr(p.bad_page, YALIS_FLAG_BAD_PAGE);
    return;
  }
  T* dst = reinterpret_cast<T*>(is_v ? p.pv_pool : p.pk_pool) + entry * width;
  const int first = pos - p.pool + 1, slot = first % p.page_size;
  const float count = (float)p.pool;
  if (slot + p.pool <= p.page_size && (width & 3) == 0 && (((uintptr_t)rows | (uintptr_t)p.pk_pool | (uintptr_t)p.pv_pool) & 15) == 0) {
    // the block lies in one page: its rows follow one another, four values a lane, eight rows in flight
    const long long row = paged_row(table, p.table_width, p.page_size, p.num_pages, p.nk, head, first);
    if (row < 0) {
      if (lane == 0 && p.bad_page) atomicOr(p.bad_page, YALIS_FLAG_BAD_PAGE);
      return;
    }
    for (int d = lane * 4; d < width; d += 128) {
      const T* src = rows + row * width + d;
      float4 sum = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int j0 = 0; j0 < p.pool; j0 += 8) {
        float4 x[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) x[j] = j0 + j < p.pool ? load4_f32(src + (j0 + j) * width) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          sum.x += x[j].x; sum.y += x[j].y; sum.z += x[j].z; sum.w += x[j].w;
        }
      }
      store4(dst + d, make_float4(sum.x / count, sum.y / count, sum.z / count, sum.w / count));
    }
    return;
  }
  for (int d0 = 0; d0 < width; d0 += 128) {      // up to four sizes a lane at a time
    float sum[4] = {0.f, 0.f, 0.f, 0.f};
    for (int at = first; at <= pos; ++at) {
      const long long row = paged_row(table, p.table_width, p.page_size, p.num_pages, p.nk, head, at);
      if (row < 0) {
        if (lane == 0 && p.bad_page) atomicOr(p.bad_page, YALIS_FLAG_BAD_PAGE);
        return;
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int d = d0 + lane + 32 * i;
        if (d < width) sum[i] += to_f32<T>(rows[row * width + d]);
      }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int d = d0 + lane + 32 * i;
      if (d < width) dst[d] = from_f32<T>(sum[i] / count);
    }
  }
}

// For steps in which a request brings several tokens: after qkv_prepare has stored them, a warp per (tile of 32 or fewer
// tokens, key or value head) looks for the tokens of its tile that end a block and stores those blocks' means.
template <typename T>
__global__ void store_block_means_kernel(const PrepParams p, int n_tokens, int tile) {
  pdl_launch_dependents();
  pdl_wait();
  const int head = blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (head >= 2 * p.nk) return;
  const int n = blockIdx.x * tile + lane;
  const bool mine = lane < tile && n < n_tokens;
  const int req = mine ? p.req_of_token[n] : -1;
  const int pos = req >= 0 ? p.positions[n] : 0;
  unsigned ends = __ballot_sync(0xffffffffu, req >= 0 && (pos + 1) % p.pool == 0);
  while (ends) {
    const int at = __ffs(ends) - 1;
    ends &= ends - 1;
    store_block_mean<T>(p, __shfl_sync(0xffffffffu, req, at), __shfl_sync(0xffffffffu, pos, at),
                        head >= p.nk ? head - p.nk : head, head >= p.nk, lane);
  }
}

// Sum over the block of the squares of `count` values (plus a bias) of a row.
template <typename T, bool VEC>
__device__ __forceinline__ float row_squares(const T* row, const T* bias, int count, float* scratch) {
  float ss = 0.f;
  if constexpr (VEC) {
    for (int c = threadIdx.x * 4; c < count; c += blockDim.x * 4) {
      float4 x = load4_f32(row + c);
      if (bias) {
        const float4 b = load4_f32(bias + c);
        x.x += b.x; x.y += b.y; x.z += b.z; x.w += b.w;
      }
      ss += (x.x * x.x + x.y * x.y) + (x.z * x.z + x.w * x.w);
    }
  } else {
    for (int c = threadIdx.x; c < count; c += blockDim.x) {
      float x = to_f32<T>(row[c]);
      if (bias) x += to_f32<T>(bias[c]);
      ss = __fmaf_rn(x, x, ss);
    }
  }
  return block_sum(ss, scratch);
}

// One warp per (token, head): heads [0, nq) are queries, then nk * maps keys, then nk values.  A warp goes on
// to further heads of its token where the grid has fewer warps than heads.
// TABLE: the block computes the token's sines and cosines once, in shared memory (steps of many tokens, where a block
// walks all heads).  VEC: four consecutive values at a time (every row, size and offset a multiple of four, aligned).
template <typename T, typename TO, bool TABLE, bool VEC>
__global__ void __launch_bounds__(256, 5) qkv_prepare_kernel(const PrepParams p) {
  extern __shared__ __align__(16) float xs_all[];   // a row of `row_floats` per warp, then (TABLE) cosines and sines
  __shared__ float scratch[32];
  pdl_launch_dependents();
  pdl_wait();
  const int n = blockIdx.x, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  const int row_floats = ((p.dim > p.vdim ? p.dim : p.vdim) + 3) & ~3;
  float* xs = xs_all + (size_t)(threadIdx.x >> 5) * row_floats;
  const int req = p.req_of_token[n];
  if (req < 0) return;
  const int pos = p.positions[n];
  const T* row = reinterpret_cast<const T*>(p.src) + (size_t)n * p.src_stride;
  const int half = p.inv_freq ? p.rot_dims >> 1 : 0;
  float* cos_s = xs_all + (size_t)warps * row_floats;
  float* sin_s = cos_s + ((half + 3) & ~3);
  if constexpr (TABLE) {
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
      float sn, cs;
      sincosf((float)pos * p.inv_freq[i], &sn, &cs);
      cos_s[i] = cs * p.rot_scale;
      sin_s[i] = sn * p.rot_scale;
    }
    __syncthreads();
  }
  float all_q = 1.f, all_k = 1.f;             // norm over all heads: 1 / root mean square of the whole of q and of k
  if (p.norm_all) {
    if (p.q_norm) all_q = 1.0f / sqrtf(row_squares<T, VEC>(row + p.q_off, reinterpret_cast<const T*>(p.q_bias), p.nq * p.dim, scratch) /
                                           (float)(p.nq * p.dim) + p.norm_eps);
    if (p.k_norm) all_k = 1.0f / sqrtf(row_squares<T, VEC>(row + p.k_off, reinterpret_cast<const T*>(p.k_bias), p.nk * p.maps * p.dim, scratch) /
                                           (float)(p.nk * p.maps * p.dim) + p.norm_eps);
  }
  auto turned = [&](int i, float& cs, float& sn) {
    if constexpr (TABLE) {
      cs = cos_s[i];
      sn = sin_s[i];
    } else {
      sincosf((float)pos * p.inv_freq[i], &sn, &cs);
      cs *= p.rot_scale;
      sn *= p.rot_scale;
    }
  };
  // what all heads of the token share: its cached row (of head 0), the query's factor, whether it ends a block
  const long long row0 = p.k_pool != nullptr ? paged_row(p.block_table + (size_t)req * p.table_width, p.table_width, p.page_size,
                                                         p.num_pages, p.nk, 0, pos)
                                             : 0;
  const float q_factor = p.q_temp_every > 0 ? p.q_scale * (1.0f + p.q_temp_coef * logf((float)((pos + 1) / p.q_temp_every + 1)))
                                            : p.q_scale;
  const bool ends_block = p.pool > 0 && (pos + 1) % p.pool == 0;
  const int keys = p.nk * p.maps;
  for (int head = blockIdx.y * warps + (threadIdx.x >> 5); head < p.nq + keys + p.nk; head += gridDim.y * warps) {
    const bool is_q = head < p.nq, is_v = head >= p.nq + keys;
    const int hh = is_q ? head : (is_v ? head - p.nq - keys : head - p.nq);
    const int width = is_v ? p.vdim : p.dim;
    const T* src = row + (is_q ? p.q_off : (is_v ? p.v_off : p.k_off)) + (size_t)hh * width;
    const T* bias = reinterpret_cast<const T*>(is_q ? p.q_bias : (is_v ? p.v_bias : p.k_bias));
    if (bias) bias += (size_t)hh * width;
    TO* dst;
    if (is_q) {
      dst = reinterpret_cast<TO*>(p.q_out) + (size_t)n * p.q_out_stride + (size_t)hh * width;
    } else if (p.k_pool != nullptr) {
      if (row0 < 0) {
        if (lane == 0 && p.bad_page) atomicOr(p.bad_page, YALIS_FLAG_BAD_PAGE);
        continue;
      }
      if (is_v) dst = reinterpret_cast<TO*>(p.v_pool) + (row0 + (long long)hh * p.page_size) * width;
      else dst = reinterpret_cast<TO*>(p.k_pool) + (row0 + (long long)(hh / p.maps) * p.page_size) * (p.maps * width) + hh % p.maps * width;
    } else {
      if (p.k_out == nullptr) continue;            // nothing keeps this layer's keys and values: queries only
      dst = is_v ? reinterpret_cast<TO*>(p.v_out) + (size_t)n * p.v_out_stride + (size_t)hh * width
                 : reinterpret_cast<TO*>(p.k_out) + (size_t)n * p.k_out_stride + (size_t)hh * width;
    }
    const float* nw = is_v ? nullptr : (is_q ? p.q_norm : p.k_norm);
    if (nw && p.norm_all) nw += (size_t)hh * width;
    const float factor = is_q ? q_factor : p.k_scale;
    __syncwarp();                                  // the warp is done with the row of its last head
    float ss = 0.f;
    if constexpr (VEC) {
      for (int d = lane * 4; d < width; d += 128) {
        float4 x = load4_f32(src + d);
        if (bias) {
          const float4 b = load4_f32(bias + d);
          x.x += b.x; x.y += b.y; x.z += b.z; x.w += b.w;
        }
        if (is_v) store4(dst + d, x);
        else *reinterpret_cast<float4*>(xs + d) = x;
        ss += (x.x * x.x + x.y * x.y) + (x.z * x.z + x.w * x.w);
      }
    } else {
      for (int d = lane; d < width; d += 32) {
        float x = to_f32<T>(src[d]);
        if (bias) x += to_f32<T>(bias[d]);
        if (is_v) dst[d] = from_f32<TO>(x);
        else xs[d] = x;
        ss = __fmaf_rn(x, x, ss);
      }
    }
    if (!is_v) {
      if (nw) {
        const float r = p.norm_all ? (is_q ? all_q : all_k) : 1.0f / sqrtf(warp_sum(ss) / (float)width + p.norm_eps);
        if constexpr (VEC) {
          for (int d = lane * 4; d < width; d += 128) {
            const float4 w = load4_f32(nw + d), x = *reinterpret_cast<const float4*>(xs + d);
            *reinterpret_cast<float4*>(xs + d) = make_float4(x.x * r * w.x, x.y * r * w.y, x.z * r * w.z, x.w * r * w.w);
          }
        } else {
          for (int d = lane; d < width; d += 32) xs[d] = xs[d] * r * nw[d];
        }
      }
      __syncwarp();
      if constexpr (VEC) {
        if (p.rot_interleaved) {
          for (int d = lane * 4; d < 2 * half; d += 128) {
            const float4 x = *reinterpret_cast<const float4*>(xs + d);
            float4 o;
            float cs, sn;
            turned(d >> 1, cs, sn);
            rotate_pair(x.x, x.y, cs, sn, o.x, o.y);
            turned((d >> 1) + 1, cs, sn);
            rotate_pair(x.z, x.w, cs, sn, o.z, o.w);
            store4(dst + d, make_float4(o.x * factor, o.y * factor, o.z * factor, o.w * factor));
          }
        } else {
          // two pairs a lane: a rotation of 64 sizes keeps the whole warp busy
          for (int i = lane * 2; i < half; i += 64) {
            const float2 a = *reinterpret_cast<const float2*>(xs + i), b = *reinterpret_cast<const float2*>(xs + i + half);
            float2 oa, ob;
            float cs, sn;
            turned(i, cs, sn);
            rotate_pair(a.x, b.x, cs, sn, oa.x, ob.x);
            turned(i + 1, cs, sn);
            rotate_pair(a.y, b.y, cs, sn, oa.y, ob.y);
            store2(dst + i, make_float2(oa.x * factor, oa.y * factor));
            store2(dst + i + half, make_float2(ob.x * factor, ob.y * factor));
          }
        }
        for (int d = 2 * half + lane * 4; d < width; d += 128) {
          const float4 x = *reinterpret_cast<const float4*>(xs + d);
          store4(dst + d, make_float4(x.x * factor, x.y * factor, x.z * factor, x.w * factor));
        }
      } else {
        for (int i = lane; i < half; i += 32) {
          float sn, cs, o1, o2;
          turned(i, cs, sn);
          const int a = p.rot_interleaved ? 2 * i : i, b = p.rot_interleaved ? 2 * i + 1 : i + half;
          rotate_pair(xs[a], xs[b], cs, sn, o1, o2);
          dst[a] = from_f32<TO>(o1 * factor);
          dst[b] = from_f32<TO>(o2 * factor);
        }
        for (int d = 2 * half + lane; d < width; d += 32) dst[d] = from_f32<TO>(xs[d] * factor);
      }
    }
    if (ends_block && !is_q) {
      __syncwarp();                                // the row that this warp has just stored ends a block
      store_block_mean<TO>(p, req, pos, hh, is_v, lane);
    }
  }
}

// The same where nothing turns and nothing is averaged: heads that are normed one by one or not at all, biases aside.  L
// lanes take a head, NV times four values each (4 L NV covers the widest head), so heads of few sizes do not leave most of
// a warp idle; the values stay in registers.  Groups of lanes are dealt to (token, head) pairs in order.
template <typename T, typename TO, int L, int NV>
__global__ void __launch_bounds__(256) qkv_plain_kernel(const PrepParams p, int n_tokens) {
  pdl_launch_dependents();
  pdl_wait();
  const int keys = p.nk * p.maps, heads = p.nq + keys + p.nk;
  const unsigned at = blockIdx.x * (256u / L) + threadIdx.x / L;
  const int n = (int)(at / (unsigned)heads), head = (int)(at - (unsigned)n * heads), sl = threadIdx.x % L;
  const int req = n < n_tokens ? p.req_of_token[n] : -1;
  const bool is_q = head < p.nq, is_v = head >= p.nq + keys;
  const int hh = is_q ? head : (is_v ? head - p.nq - keys : head - p.nq);
  const int width = is_v ? p.vdim : p.dim;
  TO* dst = nullptr;
  if (req >= 0) {
    if (is_q) {
      dst = reinterpret_cast<TO*>(p.q_out) + (size_t)n * p.q_out_stride + (size_t)hh * width;
    } else if (p.k_pool != nullptr) {
      const long long row = paged_row(p.block_table + (size_t)req * p.table_width, p.table_width, p.page_size, p.num_pages, p.nk,
                                      is_v ? hh : hh / p.maps, p.positions[n]);
      if (row < 0) {
        if (sl == 0 && p.bad_page) atomicOr(p.bad_page, YALIS_FLAG_BAD_PAGE);
      } else {
        dst = is_v ? reinterpret_cast<TO*>(p.v_pool) + row * width
                   : reinterpret_cast<TO*>(p.k_pool) + row * (p.maps * width) + hh % p.maps * width;
      }
    } else if (p.k_out != nullptr) {
      dst = is_v ? reinterpret_cast<TO*>(p.v_out) + (size_t)n * p.v_out_stride + (size_t)hh * width
                 : reinterpret_cast<TO*>(p.k_out) + (size_t)n * p.k_out_stride + (size_t)hh * width;
    }
  }
  const T* src = reinterpret_cast<const T*>(p.src) + (size_t)(req >= 0 ? n : 0) * p.src_stride +
                 (is_q ? p.q_off : (is_v ? p.v_off : p.k_off)) + (size_t)hh * width;
  float4 x[NV];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int d = (sl + i * L) * 4;
    x[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (dst != nullptr && d < width) x[i] = load4_f32(src + d);
    ss += (x[i].x * x[i].x + x[i].y * x[i].y) + (x[i].z * x[i].z + x[i].w * x[i].w);
  }
#pragma unroll
  for (int o = L / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  if (dst == nullptr) return;
  const float* nw = is_v ? nullptr : (is_q ? p.q_norm : p.k_norm);
  const float r = (is_v ? 1.0f : (is_q ? p.q_scale : p.k_scale)) * (nw ? 1.0f / sqrtf(ss / (float)width + p.norm_eps) : 1.0f);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int d = (sl + i * L) * 4;
    if (d >= width) continue;
    float4 w = make_float4(1.f, 1.f, 1.f, 1.f);
    if (nw) w = load4_f32(nw + d);
    store4(dst + d, make_float4(x[i].x * r * w.x, x[i].y * r * w.y, x[i].z * r * w.z, x[i].w * r * w.w));
  }
}

template <typename T, typename TO>
int launch_qkv_plain(const PrepParams& p, int n_tokens, cudaStream_t stream) {
  const int narrow = p.dim < p.vdim ? p.dim : p.vdim, widest = p.dim < p.vdim ? p.vdim : p.dim;
  const long long pairs = (long long)n_tokens * (p.nq + (p.maps + 1) * p.nk);
  if (pairs >= 1LL << 31) return YALIS_ERR_SHAPE;
  auto go = [&](auto kernel, int lanes) {
    return yalis_launch(kernel, dim3((unsigned)((pairs * lanes + 255) / 256)), dim3(256), 0, stream, p, n_tokens);
  };
  if (narrow <= 32 && widest <= 64) return go(qkv_plain_kernel<T, TO, 8, 2>, 8);
  if (narrow <= 64 && widest <= 128) return go(qkv_plain_kernel<T, TO, 16, 2>, 16);
  return go(qkv_plain_kernel<T, TO, 32, 2>, 32);
}

template <typename T, typename TO>
int launch_qkv_prepare(const PrepParams& p, dim3 grid, int warps, bool table, bool vec, cudaStream_t stream) {
  const int row_floats = ((p.dim > p.vdim ? p.dim : p.vdim) + 3) & ~3;
  size_t smem = (size_t)warps * row_floats * sizeof(float);
  if (table) smem += 2 * (size_t)((p.rot_dims / 2 + 3) & ~3) * sizeof(float);
  if (smem > 48 * 1024) return YALIS_ERR_SHAPE;
  const dim3 block(32 * warps);
  if (table) return vec ? yalis_launch(qkv_prepare_kernel<T, TO, true, true>, grid, block, smem, stream, p)
                        : yalis_launch(qkv_prepare_kernel<T, TO, true, false>, grid, block, smem, stream, p);
  return vec ? yalis_launch(qkv_prepare_kernel<T, TO, false, true>, grid, block, smem, stream, p)
             : yalis_launch(qkv_prepare_kernel<T, TO, false, false>, grid, block, smem, stream, p);
}

// ACT: 0 gelu with erf, 1 gelu with tanh, 2 silu, 3 the square of relu, 4 tanh.
// With `bias` (float32, one per column) it is added to x first.  TO: the result's type (T, or float32).
template <typename T, typename TO>
__global__ void activation_kernel(const T* __restrict__ x, int x_stride, TO* __restrict__ y, int y_stride, int rows,
                                  int cols, int act, const float* __restrict__ bias) {
  pdl_launch_dependents();
  pdl_wait();
  const size_t total = (size_t)rows * cols;
  for (size_t e = (size_t)blockIdx.x * blockDim.x + threadIdx.x; e < total; e += (size_t)gridDim.x * blockDim.x) {
    const size_t r = e / cols, c = e - r * cols;
    float z = to_f32<T>(x[r * x_stride + c]);
    if (bias) z += bias[c];
    float o;
    if (act == 0) o = 0.5f * z * (1.0f + erff(z * 0.70710678118654752440f));
    else if (act == 1) o = 0.5f * z * (1.0f + tanhf(0.79788456080286535588f * (z + 0.044715f * z * z * z)));
    else if (act == 2) o = silu_exact(z);
    else if (act == 4) o = tanhf(z);
    else o = fmaxf(z, 0.f) * fmaxf(z, 0.f);
    y[r * y_stride + c] = from_f32<TO>(o);
  }
}

// The same, eight elements a thread, for bfloat16 rows that start on 16-byte boundaries and whose width is a
// multiple of 8.  grid: (ceil(cols / 8 / 256), rows).
__device__ __forceinline__ float act_value(float z, int act) {
  if (act == 0) return 0.5f * z * (1.0f + erff(z * 0.70710678118654752440f));
  if (act == 1) return 0.5f * z * (1.0f + tanhf(0.79788456080286535588f * (z + 0.044715f * z * z * z)));
  if (act == 3) return fmaxf(z, 0.f) * fmaxf(z, 0.f);
  if (act == 4) return tanhf(z);
  return silu_exact(z);
}

__global__ void activation_bf16x8_kernel(const __nv_bfloat16* __restrict__ x, int x_stride, __nv_bfloat16* __restrict__ y,
                                         int y_stride, int cols, int act, const float* __restrict__ bias) {
  pdl_launch_dependents();
  pdl_wait();
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * 8;
  if (c >= cols) return;
  const size_t r = blockIdx.y;
  uint4 raw = *reinterpret_cast<const uint4*>(x + r * x_stride + c);
  __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    float2 z = __bfloat1622float2(h[i]);
    if (bias) {
      const float2 b = *reinterpret_cast<const float2*>(bias + c + 2 * i);
      z.x += b.x;
      z.y += b.y;
    }
    h[i] = __floats2bfloat162_rn(act_value(z.x, act), act_value(z.y, act));
  }
  *reinterpret_cast<uint4*>(y + r * y_stride + c) = raw;
}

// Four elements a thread with float32 results (bfloat16 rows on 8-byte boundaries, float32 rows on 16-byte ones).  Its
// reader may be a kernel of few, long blocks (a recurrence over the rows it makes): those are let in only once this one
// has begun, so that they do not crowd onto the SMs that come free first.
template <typename T>
__global__ void activation_f32x4_kernel(const T* __restrict__ x, int x_stride, float* __restrict__ y, int y_stride, int rows,
                                        int cols, int act, const float* __restrict__ bias) {
  pdl_wait();
  pdl_launch_dependents();
  const int quads = cols >> 2;
  const size_t total = (size_t)rows * quads;
  for (size_t e = (size_t)blockIdx.x * blockDim.x + threadIdx.x; e < total; e += (size_t)gridDim.x * blockDim.x) {
    const size_t r = e / quads;
    const int c = (int)(e - r * quads) << 2;
    float4 z = load4_f32(x + r * x_stride + c);
    if (bias) {
      const float4 b = load4_f32(bias + c);
      z.x += b.x; z.y += b.y; z.z += b.z; z.w += b.w;
    }
    store4(y + r * y_stride + c, make_float4(act_value(z.x, act), act_value(z.y, act), act_value(z.z, act), act_value(z.w, act)));
  }
}

// A gated activation over rows that hold a gate part and an up part (at column offsets of one matrix):
//   kind 0:  y = silu(g) * u
//   kind 1:  g <- min(g, limit), u <- clamp(u, -limit, limit);  y = g * sigmoid(alpha * g) * (u + shift)
// float32 arithmetic, one rounding.
template <typename T>
__global__ void gated_activation_kernel(const T* __restrict__ x, long x_stride, int gate_off, int up_off, T* __restrict__ y,
                                        long y_stride, int rows, int cols, int kind, float limit, float alpha, float shift) {
  pdl_launch_dependents();
  pdl_wait();
  const size_t total = (size_t)rows * cols;
  for (size_t e = (size_t)blockIdx.x * blockDim.x + threadIdx.x; e < total; e += (size_t)gridDim.x * blockDim.x) {
    const size_t r = e / cols, c = e - r * cols;
    float g = to_f32<T>(x[r * x_stride + gate_off + c]), u = to_f32<T>(x[r * x_stride + up_off + c]);
    float o;
    if (kind == 1) {
      g = fminf(g, limit);
      u = fminf(fmaxf(u, -limit), limit);
      o = g * (1.0f / (1.0f + expf(-alpha * g))) * (u + shift);
    } else {
      o = silu_exact(g) * u;
    }
    y[r * y_stride + c] = from_f32<T>(o);
  }
}

// The same, eight elements a thread, for bfloat16 rows whose two parts and whose results start on 16-byte boundaries
// (width and both offsets multiples of 8).  The result is rounded to 8 bits of mantissa at once, so the fast
// exponential and division do not show.  grid: (ceil(cols / 8 / 128), rows).
__global__ void gated_activation_bf16x8_kernel(const __nv_bfloat16* __restrict__ x, long x_stride, int gate_off, int up_off,
                                               __nv_bfloat16* __restrict__ y, long y_stride, int cols, int kind, float limit,
                                               float alpha, float shift) {
  pdl_launch_dependents();
  pdl_wait();
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * 8;
  if (c >= cols) return;
  const size_t r = blockIdx.y;
  uint4 graw = *reinterpret_cast<const uint4*>(x + r * x_stride + gate_off + c);
  const uint4 uraw = *reinterpret_cast<const uint4*>(x + r * x_stride + up_off + c);
  __nv_bfloat162* gh = reinterpret_cast<__nv_bfloat162*>(&graw);
  const __nv_bfloat162* uh = reinterpret_cast<const __nv_bfloat162*>(&uraw);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    float2 g = __bfloat1622float2(gh[i]);
    float2 u = __bfloat1622float2(uh[i]);
    if (kind == 1) {
      g.x = fminf(g.x, limit); g.y = fminf(g.y, limit);
      u.x = fminf(fmaxf(u.x, -limit), limit); u.y = fminf(fmaxf(u.y, -limit), limit);
      gh[i] = __floats2bfloat162_rn(__fdividef(g.x, 1.0f + __expf(-alpha * g.x)) * (u.x + shift),
                                    __fdividef(g.y, 1.0f + __expf(-alpha * g.y)) * (u.y + shift));
    } else {
      gh[i] = __floats2bfloat162_rn(silu_bf16_path(g.x) * u.x, silu_bf16_path(g.y) * u.y);
    }
  }
  *reinterpret_cast<uint4*>(y + r * y_stride + c) = graw;
}

// x[n, :] += other[n, :] + vec[:]   (either may be absent)
__global__ void add_rows_vector_kernel(float* __restrict__ x, const float* __restrict__ other,
                                       const float* __restrict__ vec, int rows, int cols) {
  pdl_launch_dependents();
  pdl_wait();
  const size_t total = (size_t)rows * cols;
  for (size_t e = (size_t)blockIdx.x * blockDim.x + threadIdx.x; e < total; e += (size_t)gridDim.x * blockDim.x) {
    float v = x[e];
    if (other) v += other[e];
    if (vec) v += vec[e % cols];
    x[e] = v;
  }
}

}  // namespace

// pool > 0: the means of blocks of `pool` keys and values go to pk_pool / pv_pool.  With single_tokens (no request brings
// more than one token) the warp that stores a block's last row does it; otherwise a second kernel does, once all rows of
// the step are stored.
// maps > 1 (without pooled blocks): every key/value head has `maps` keys of size dim, which lie side by side in src and in a
// cached row; nk counts the key/value heads.
// out_dtype: the dtype of q_out and of the plain k_out / v_out (pools always have the model dtype `dtype`).
YALIS_API int yalis_qkv_prepare(const void* src, int dtype, int src_stride, int q_off, int k_off, int v_off,
                                const void* q_bias, const void* k_bias, const void* v_bias, const float* q_norm,
                                const float* k_norm, float norm_eps, const float* inv_freq, int rot_dims,
                                int rot_interleaved, float rot_scale, int norm_all, float q_scale, float k_scale, float q_temp_coef, int q_temp_every,
                                void* q_out, int q_out_stride, void* k_out, int k_out_stride, void* v_out,
                                int v_out_stride, int out_dtype, void* k_pool, void* v_pool,
                                const int32_t* block_table, int table_width, int page_size, int num_pages,
                                const int32_t* positions, const int32_t* req_of_token, int n_tokens, int nq, int nk,
                                int dim, int vdim, int32_t* bad_page, int pool, void* pk_pool, void* pv_pool,
                                const int32_t* pool_table, int pool_table_width, int pool_page_size, int pool_num_pages,
                                int single_tokens, int maps, cudaStream_t stream) {
  if (n_tokens <= 0) return YALIS_OK;
  if (pool < 0 || (pool > 0 && (!k_pool || !pk_pool || !pv_pool || !pool_table || pool_page_size < 1))) return YALIS_ERR_SHAPE;
  if (dim <= 0 || dim > kMaxHeadDim || vdim <= 0 || vdim > kMaxHeadDim || nq <= 0 || nk <= 0 || maps < 1 ||
      nq + (maps + 1) * nk > 65535 || (maps > 1 && pool > 0))
    return YALIS_ERR_SHAPE;
  if (inv_freq && (rot_dims <= 0 || (rot_dims & 1) || rot_dims > dim)) return YALIS_ERR_SHAPE;
  if (k_pool && out_dtype != dtype) return YALIS_ERR_DTYPE;
  PrepParams p;
  p.src = src; p.src_stride = src_stride; p.q_off = q_off; p.k_off = k_off; p.v_off = v_off;
  p.q_bias = q_bias; p.k_bias = k_bias; p.v_bias = v_bias; p.q_norm = q_norm; p.k_norm = k_norm; p.norm_eps = norm_eps;
  p.inv_freq = inv_freq; p.rot_dims = rot_dims; p.rot_interleaved = rot_interleaved;
  p.rot_scale = rot_scale; p.norm_all = norm_all; p.q_scale = q_scale; p.k_scale = k_scale;
  p.q_temp_coef = q_temp_coef; p.q_temp_every = q_temp_every;
  p.q_out = q_out; p.q_out_stride = q_out_stride; p.k_out = k_out; p.k_out_stride = k_out_stride;
  p.v_out = v_out; p.v_out_stride = v_out_stride; p.k_pool = k_pool; p.v_pool = v_pool; p.block_table = block_table;
  p.table_width = table_width; p.page_size = page_size; p.num_pages = num_pages; p.positions = positions;
  p.req_of_token = req_of_token; p.nq = nq; p.nk = nk; p.dim = dim; p.vdim = vdim; p.maps = maps; p.bad_page = bad_page;
  p.pool = single_tokens ? pool : 0;
  p.pk_pool = pk_pool; p.pv_pool = pv_pool; p.pool_table = pool_table; p.pool_table_width = pool_table_width;
  p.pool_page_size = pool_page_size; p.pool_num_pages = pool_num_pages;
  // Steps of many tokens: a block of eight warps walks all heads of its token, which shares the sines and cosines and
  // the sums of a norm over all heads.  Few tokens: four heads a block, so that more blocks run at once.
  const bool per_token = n_tokens >= 2 * yalis_sm_count() && dim <= 512 && vdim <= 512;
  const int warps = per_token ? 8 : 4;
  const dim3 grid(n_tokens, per_token ? 1 : (nq + (maps + 1) * nk + warps - 1) / warps);
  const bool table = per_token && inv_freq != nullptr;
  const uintptr_t ptrs = (uintptr_t)src | (uintptr_t)q_bias | (uintptr_t)k_bias | (uintptr_t)v_bias | (uintptr_t)q_norm |
                         (uintptr_t)k_norm | (uintptr_t)q_out | (uintptr_t)k_out | (uintptr_t)v_out | (uintptr_t)k_pool |
                         (uintptr_t)v_pool;
  const bool vec = ((dim | vdim | rot_dims | src_stride | q_off | k_off | v_off | q_out_stride | k_out_stride | v_out_stride) & 3) == 0 &&
                   (ptrs & 15) == 0;
  int st;
  const bool plain = vec && !inv_freq && !norm_all && q_temp_every <= 0 && pool == 0 && !q_bias && !k_bias && !v_bias &&
                     dim <= 256 && vdim <= 256;
  if (plain && dtype == YALIS_F32 && out_dtype == YALIS_F32) return launch_qkv_plain<float, float>(p, n_tokens, stream);
  if (plain && dtype == YALIS_BF16 && out_dtype == YALIS_BF16)
    return launch_qkv_plain<__nv_bfloat16, __nv_bfloat16>(p, n_tokens, stream);
  if (plain && dtype == YALIS_BF16 && out_dtype == YALIS_F32) return launch_qkv_plain<__nv_bfloat16, float>(p, n_tokens, stream);
  if (dtype == YALIS_F32 && out_dtype == YALIS_F32) st = launch_qkv_prepare<float, float>(p, grid, warps, table, vec, stream);
  else if (dtype == YALIS_BF16 && out_dtype == YALIS_BF16)
    st = launch_qkv_prepare<__nv_bfloat16, __nv_bfloat16>(p, grid, warps, table, vec, stream);
  else if (dtype == YALIS_BF16 && out_dtype == YALIS_F32)
    st = launch_qkv_prepare<__nv_bfloat16, float>(p, grid, warps, table, vec, stream);
  else
    return YALIS_ERR_DTYPE;
  if (st != YALIS_OK || pool == 0 || single_tokens) return st;
  p.pool = pool;
  const int tile = pool < 32 ? pool : 32;         // about one block's end per tile
  const dim3 means((n_tokens + tile - 1) / tile, (2 * nk + 3) / 4);
  YALIS_DISPATCH_DTYPE(dtype, T, return yalis_launch(store_block_means_kernel<T>, means, dim3(128), 0, stream, p, n_tokens, tile));
  return YALIS_OK;
}

// y_f32: the result is float32 whatever the input's type.
YALIS_API int yalis_activation(const void* x, int x_stride, void* y, int y_stride, int dtype, int y_f32, int rows, int cols,
                               int act, const float* bias, cudaStream_t stream) {
  if (rows <= 0 || cols <= 0) return YALIS_OK;
  if (act < 0 || act > 4) return YALIS_ERR_SHAPE;
  const size_t total = (size_t)rows * cols;
  const int blocks = (int)((total + 255) / 256 < 148 * 16 ? (total + 255) / 256 : 148 * 16);
  if (y_f32 && cols % 4 == 0 && x_stride % 4 == 0 && y_stride % 4 == 0 && !((uintptr_t)x & (dtype == YALIS_BF16 ? 7 : 15)) &&
      !(((uintptr_t)y | (uintptr_t)bias) & 15)) {
    const size_t quads = (total / 4 + 255) / 256;
    const dim3 grid((unsigned)(quads < 148 * 16 ? quads : 148 * 16));
    YALIS_DISPATCH_DTYPE(dtype, T, return yalis_launch(activation_f32x4_kernel<T>, grid, dim3(256), 0, stream, (const T*)x,
                                                       x_stride, (float*)y, y_stride, rows, cols, act, bias));
  }
  if (y_f32 && dtype == YALIS_BF16)
    return yalis_launch(activation_kernel<__nv_bfloat16, float>, dim3(blocks), dim3(256), 0, stream, (const __nv_bfloat16*)x,
                        x_stride, (float*)y, y_stride, rows, cols, act, bias);
  if (dtype == YALIS_BF16 && cols % 8 == 0 && x_stride % 8 == 0 && y_stride % 8 == 0 && !((uintptr_t)x & 15) &&
      !((uintptr_t)y & 15) && !((uintptr_t)bias & 7) && rows <= 65535)
    return yalis_launch(activation_bf16x8_kernel, dim3((cols / 8 + 127) / 128, rows), dim3(128), 0, stream,
                        (const __nv_bfloat16*)x, x_stride, (__nv_bfloat16*)y, y_stride, cols, act, bias);
  YALIS_DISPATCH_DTYPE(dtype, T,
                       return yalis_launch((activation_kernel<T, T>), dim3(blocks), dim3(256), 0, stream, (const T*)x, x_stride,
                                           (T*)y, y_stride, rows, cols, act, bias));
  return YALIS_OK;
}

YALIS_API int yalis_gated_activation(const void* x, long long x_stride, int gate_off, int up_off, void* y, long long y_stride,
                                     int dtype, int rows, int cols, int kind, float limit, float alpha, float shift,
                                     cudaStream_t stream) {
  if (rows <= 0 || cols <= 0) return YALIS_OK;
  if (kind < 0 || kind > 1) return YALIS_ERR_SHAPE;
  if (dtype == YALIS_BF16 && cols % 8 == 0 && x_stride % 8 == 0 && y_stride % 8 == 0 && gate_off % 8 == 0 && up_off % 8 == 0 &&
      !((uintptr_t)x & 15) && !((uintptr_t)y & 15) && rows <= 65535)
    return yalis_launch(gated_activation_bf16x8_kernel, dim3((cols / 8 + 127) / 128, rows), dim3(128), 0, stream,
                        (const __nv_bfloat16*)x, (long)x_stride, gate_off, up_off, (__nv_bfloat16*)y, (long)y_stride, cols, kind,
                        limit, alpha, shift);
  const size_t total = (size_t)rows * cols;
  const int blocks = (int)((total + 255) / 256 < 148 * 16 ? (total + 255) / 256 : 148 * 16);
  YALIS_DISPATCH_DTYPE(dtype, T,
                       return yalis_launch(gated_activation_kernel<T>, dim3(blocks), dim3(256), 0, stream, (const T*)x,
                                           (long)x_stride, gate_off, up_off, (T*)y, (long)y_stride, rows, cols, kind, limit,
                                           alpha, shift));
  return YALIS_OK;
}

YALIS_API int yalis_add_rows_vector(float* x, const float* other, const float* vec, int rows, int cols,
                                    cudaStream_t stream) {
  if (rows <= 0 || cols <= 0) return YALIS_OK;
  const size_t total = (size_t)rows * cols;
  const int blocks = (int)((total + 255) / 256 < 148 * 16 ? (total + 255) / 256 : 148 * 16);
  return yalis_launch(add_rows_vector_kernel, dim3(blocks), dim3(256), 0, stream, x, other, vec, rows, cols);
}
