// Attention through low-rank latents.  A token's keys and values of all heads are functions of
// one latent vector c (kv_rank numbers) and one rotated key part shared by the heads (rot_dim
// numbers); the cache holds just these, as one key row [c | rotated part] of kv_rank + rot_dim
// channels.  The heads' key and value maps are folded to the query's and the output's side:
//   score_h = (U_k,h^T q_h) . c + q_rot,h . k_rot          out_h = U_v,h (sum_j p_j c_j)
// so attention runs as one shared key head whose values are the first kv_rank channels of its keys.
// This file holds what goes before that attention: the norms of the two latents, the rotation
// of adjacent pairs (2i, 2i + 1) and the write into the paged cache.  Everything is computed in 32-bit from the
// 32-bit results of the projections and rounded once.
#include "common.cuh"

namespace {
// Where a row's key goes: the first of its channels inside a plane of the paged cache.
__device__ __forceinline__ size_t key_offset(const int* __restrict__ block_table, int table_stride, int slot, int pos,
                                             int page_size, long long page_stride, int hd) {
  const int page = block_table[(size_t)slot * table_stride + pos / page_size];
  return (size_t)page * page_stride + (size_t)(pos % page_size) * hd;
}

// Channel j of a rotated part v (pairs (2i, 2i + 1), the first rot_half of them turned).
__device__ __forceinline__ float turned(const float* v, int j, int rot_dim, const float2* __restrict__ cos_sin,
                                        int rot_half) {
  const int i = j >> 1;
  if (!cos_sin || i >= rot_half) return v[j];
  const float2 cs = cos_sin[i];
  const float a = v[2 * i], b = v[2 * i + 1];
  return (j & 1) ? fmaf(b, cs.x, a * cs.y) : fmaf(a, cs.x, -b * cs.y);
}

// The key row of one token by a whole block: c[0:kv_rank] normed (gain wc) into the K plane and, the
// same values, the V plane (null: none), c[kv_rank : kv_rank + rot_dim] turned behind it.
template <typename T>
__device__ __forceinline__ void store_key_row(const float* c, const float* __restrict__ wc,
                                              const float2* __restrict__ cos_sin, int rot_half, T* __restrict__ k_row,
                                              T* __restrict__ v_row, int kv_rank, int rot_dim, float eps,
                                              float* scratch) {
  const int tid = threadIdx.x;
  float ss = 0.f;
  for (int i = tid; i < kv_rank; i += blockDim.x) ss = fmaf(c[i], c[i], ss);
  ss = block_sum(ss, scratch);
  const float sc = 1.0f / sqrtf(ss / (float)kv_rank + eps);
  for (int i = tid; i < kv_rank; i += blockDim.x) {
    const T v = from_f32<T>(c[i] * sc * wc[i]);
    k_row[i] = v;
    if (v_row) v_row[i] = v;
  }
  for (int j = tid; j < rot_dim; j += blockDim.x)
    k_row[kv_rank + j] = from_f32<T>(turned(c + kv_rank, j, rot_dim, cos_sin, rot_half));
}

// One block per row.  proj[row] = [ query latent (q_rank) | key-value latent (kv_rank) | key part
// to rotate (rot_dim) ].  The query latent is normed (gain wq) into cq_out; the key-value latent
// is normed (gain wc) into the row's place in the K plane and, the same values, the V plane (null:
// the cache has none, values are read from the key rows);
// the key part is rotated by the row's angles (cos_sin[row][i] = (cos, sin) of angle i, the first
// rot_half pairs; null: no rotation) and written behind the latent in the K plane.  The V plane's
// channels behind the latent are never written and stay zero.  clear_proj: the row of proj that
// was read is zeroed at the end (it lies in a buffer that a split-K product adds into).
template <typename T>
__global__ void __launch_bounds__(512) latent_store_kernel(
    float* __restrict__ proj, int proj_stride, const float* __restrict__ wq, const float* __restrict__ wc,
    const float2* __restrict__ cos_sin, int rot_half, T* __restrict__ cq_out, T* __restrict__ k_plane,
    T* __restrict__ v_plane, long long page_stride, const int* __restrict__ block_table, int table_stride,
    const int* __restrict__ row_slot, const int* __restrict__ row_pos, int page_size, int q_rank, int kv_rank,
    int rot_dim, float eps, int write_cache, int clear_proj) {
  __shared__ float scratch[33];
  pdl_trigger();
  pdl_wait();
  const int r = blockIdx.x, tid = threadIdx.x;
  float* p = proj + (size_t)r * proj_stride;
  float ss = 0.f;
  for (int i = tid; i < q_rank; i += blockDim.x) ss = fmaf(p[i], p[i], ss);
  ss = block_sum(ss, scratch);
  const float sq = 1.0f / sqrtf(ss / (float)q_rank + eps);
  for (int i = tid; i < q_rank; i += blockDim.x)
    cq_out[(size_t)r * q_rank + i] = from_f32<T>(p[i] * sq * wq[i]);
  if (!write_cache) {
    if (clear_proj) {
      __syncthreads();
      for (int i = tid; i < q_rank + kv_rank + rot_dim; i += blockDim.x) p[i] = 0.f;
    }
    return;
  }
  const size_t off = key_offset(block_table, table_stride, row_slot[r], row_pos[r], page_size, page_stride,
                                kv_rank + rot_dim);
  store_key_row<T>(p + q_rank, wc, cos_sin ? cos_sin + (size_t)r * rot_half : nullptr, rot_half, k_plane + off,
                   v_plane ? v_plane + off : nullptr, kv_rank, rot_dim, eps, scratch);
  if (clear_proj) {
    __syncthreads();
    for (int i = tid; i < q_rank + kv_rank + rot_dim; i += blockDim.x) p[i] = 0.f;
  }
}

// q[row][h] = [ plain part (dim) | part to rotate (rot_dim) ] in 32-bit.  The plain part is rounded
// into q_plain[row][h][0:dim] (the operand of the product with U_k,h); the rotated part goes to
// q_full[row][h][kv_rank : kv_rank + rot_dim], behind the place of that product's result.  A pair
// of the rotated part is one thread's work (both values read, both written).  clear: what was
// read of q is zeroed.
template <typename T>
__global__ void latent_query_kernel(float* __restrict__ q, int q_stride, const float2* __restrict__ cos_sin,
                                    int rot_half, T* __restrict__ q_plain, T* __restrict__ q_full, long long total,
                                    int H, int dim, int rot_dim, int kv_rank, int clear) {
  pdl_trigger();
  pdl_wait();
  const int per_head = dim + rot_dim, hd = kv_rank + rot_dim;
  for (long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x; idx < total;
       idx += (long long)gridDim.x * blockDim.x) {
    const long long rh = idx / per_head;
    const int e = (int)(idx - rh * per_head);
    const long long r = rh / H;
    const int h = (int)(rh - r * H);
    float* src = q + (size_t)r * q_stride + (size_t)h * per_head;
    if (e < dim) {
      q_plain[(size_t)rh * dim + e] = from_f32<T>(src[e]);
      if (clear) src[e] = 0.f;
    } else {
      const int j = e - dim, i = j >> 1;
      if (j & 1) continue;                       // the pair's even member does both
      const bool two = j + 1 < rot_dim;
      const float a = src[e], b = two ? src[e + 1] : 0.f;
      float va = a, vb = b;
      if (cos_sin && i < rot_half) {
        const float2 cs = cos_sin[(size_t)r * rot_half + i];
        va = fmaf(a, cs.x, -b * cs.y);
        vb = fmaf(b, cs.x, a * cs.y);
      }
      T* dst = q_full + (size_t)rh * hd + kv_rank + j;
      dst[0] = from_f32<T>(va);
      if (two) dst[1] = from_f32<T>(vb);
      if (clear) {
        src[e] = 0.f;
        if (two) src[e + 1] = 0.f;
      }
    }
  }
}
// The same with four channels per thread and accesses of 16 and 8 bytes: dim, rot_dim, kv_rank and
// the row stride multiples of four, every base aligned.
template <typename T> __device__ __forceinline__ void put4(T* dst, float a, float b, float c, float d);
template <> __device__ __forceinline__ void put4<float>(float* dst, float a, float b, float c, float d) {
  *reinterpret_cast<float4*>(dst) = make_float4(a, b, c, d);
}
template <> __device__ __forceinline__ void put4<bf16>(bf16* dst, float a, float b, float c, float d) {
  const __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d);
  *reinterpret_cast<uint2*>(dst) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
}
// channels e .. e + 3 of the query `q` [dim plain | rot_dim to rotate] of (row, head) rh
template <typename T>
__device__ __forceinline__ void query_piece(float* q, int e, size_t rh, const float2* __restrict__ cos_sin,
                                            int rot_half, T* __restrict__ q_plain, T* __restrict__ q_full, int dim,
                                            int rot_dim, int kv_rank, int clear) {
  float4* src = reinterpret_cast<float4*>(q + e);
  float4 v = *src;
  if (clear) *src = make_float4(0.f, 0.f, 0.f, 0.f);
  if (e < dim) {
    put4<T>(q_plain + rh * dim + e, v.x, v.y, v.z, v.w);
    return;
  }
  const int j = e - dim, i = j >> 1;
  if (cos_sin) {
    if (i < rot_half) {
      const float2 cs = cos_sin[i];
      const float a = v.x, b = v.y;
      v.x = fmaf(a, cs.x, -b * cs.y), v.y = fmaf(b, cs.x, a * cs.y);
    }
    if (i + 1 < rot_half) {
      const float2 cs = cos_sin[i + 1];
      const float a = v.z, b = v.w;
      v.z = fmaf(a, cs.x, -b * cs.y), v.w = fmaf(b, cs.x, a * cs.y);
    }
  }
  put4<T>(q_full + rh * (kv_rank + rot_dim) + kv_rank + j, v.x, v.y, v.z, v.w);
}
template <typename T>
__global__ void __launch_bounds__(256) latent_query_vec_kernel(float* __restrict__ q, int q_stride,
                                                               const float2* __restrict__ cos_sin, int rot_half,
                                                               T* __restrict__ q_plain, T* __restrict__ q_full,
                                                               unsigned total, int H, int dim, int rot_dim,
                                                               int kv_rank, int clear) {
  pdl_trigger();
  pdl_wait();
  const unsigned per_head = (unsigned)(dim + rot_dim) >> 2;
  for (unsigned idx = blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += gridDim.x * blockDim.x) {
    const unsigned rh = idx / per_head, r = rh / (unsigned)H, h = rh - r * H;
    query_piece<T>(q + (size_t)r * q_stride + (size_t)h * (dim + rot_dim), (int)(idx - rh * per_head) * 4, rh,
                   cos_sin ? cos_sin + (size_t)r * rot_half : nullptr, rot_half, q_plain, q_full, dim, rot_dim,
                   kv_rank, clear);
  }
}

// Both in one launch, for queries that come straight from the mixer's input: proj[row] holds the
// heads' queries from column q_col on and [latent (kv_rank) | key part to rotate (rot_dim)] from
// column c_col on.  grid (rows, 1 + shares): the first block of a row writes its key row, the others
// share its queries.  VEC: as latent_query_vec_kernel, else pairs.
struct PrepareArgs {
  float* proj; int proj_stride, q_col, c_col;
  const float* wc;
  const float2* cos_sin; int rot_half;
  long long page_stride;
  const int *block_table, *row_slot, *row_pos;
  int table_stride, page_size, H, dim, rot_dim, kv_rank;
  float eps;
  int write_cache, clear;
};
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) latent_prepare_kernel(const PrepareArgs a, T* __restrict__ q_plain,
                                                             T* __restrict__ q_full, T* __restrict__ k_plane,
                                                             T* __restrict__ v_plane) {
  __shared__ float scratch[33];
  pdl_trigger();
  pdl_wait();
  const int r = blockIdx.x, per_head = a.dim + a.rot_dim, hd = a.kv_rank + a.rot_dim;
  float* p = a.proj + (size_t)r * a.proj_stride;
  const float2* cs = a.cos_sin ? a.cos_sin + (size_t)r * a.rot_half : nullptr;
  if (blockIdx.y == 0) {
    float* c = p + a.c_col;
    if (a.write_cache) {
      const size_t off = key_offset(a.block_table, a.table_stride, a.row_slot[r], a.row_pos[r], a.page_size,
                                    a.page_stride, hd);
      store_key_row<T>(c, a.wc, cs, a.rot_half, k_plane + off, v_plane ? v_plane + off : nullptr, a.kv_rank,
                       a.rot_dim, a.eps, scratch);
    }
    if (a.clear) {
      __syncthreads();
      for (int i = threadIdx.x; i < hd; i += blockDim.x) c[i] = 0.f;
    }
    return;
  }
  const int first = (blockIdx.y - 1) * blockDim.x + threadIdx.x, step = (gridDim.y - 1) * blockDim.x;
  if (VEC) {
    for (int idx = first; idx < a.H * (per_head >> 2); idx += step) {
      const int h = idx / (per_head >> 2), e = (idx - h * (per_head >> 2)) * 4;
      query_piece<T>(p + a.q_col + (size_t)h * per_head, e, (size_t)r * a.H + h, cs, a.rot_half, q_plain, q_full,
                     a.dim, a.rot_dim, a.kv_rank, a.clear);
    }
    return;
  }
  for (int idx = first; idx < a.H * per_head; idx += step) {
    const int h = idx / per_head, e = idx - h * per_head;
    const size_t rh = (size_t)r * a.H + h;
    float* src = p + a.q_col + (size_t)h * per_head;
    if (e < a.dim) {
      q_plain[rh * a.dim + e] = from_f32<T>(src[e]);
      if (a.clear) src[e] = 0.f;
    } else if (!((e - a.dim) & 1)) {             // a pair is one thread's work
      const int j = e - a.dim, n = a.rot_dim - j < 2 ? 1 : 2;
      float v[2];
      for (int i = 0; i < n; ++i) v[i] = turned(src + a.dim, j + i, a.rot_dim, cs, a.rot_half);
      for (int i = 0; i < n; ++i) {
        q_full[rh * hd + a.kv_rank + j + i] = from_f32<T>(v[i]);
        if (a.clear) src[e + i] = 0.f;
      }
    }
  }
}
}  // namespace

LLM_EXPORT int llm_latent_store(float* proj, int proj_stride, const float* wq, const float* wc,
                                const float* cos_sin, int rot_half, void* cq_out, void* k_plane, void* v_plane,
                                int dtype, long long page_stride, const int* block_table, int table_stride,
                                const int* row_slot, const int* row_pos, int rows, int page_size, int q_rank,
                                int kv_rank, int rot_dim, float eps, int write_cache, int clear_proj,
                                cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (q_rank <= 0 || kv_rank <= 0 || rot_dim < 0 || 2 * rot_half > rot_dim) return LLM_ERR_ARGUMENT;
  // few rows: a row is a chain of round trips to memory, shorter with more threads
  const int most = rows < 512 ? 512 : 256, longest = q_rank > kv_rank ? q_rank : kv_rank;
  const int threads = longest >= most ? most : longest > 128 ? (longest + 31) / 32 * 32 : 128;
  if (dtype == LLM_F32)
    return launched_many_blocks(launch_pdl(latent_store_kernel<float>, rows, threads, 0, stream, proj, proj_stride, wq, wc,
                      (const float2*)cos_sin, rot_half, (float*)cq_out, (float*)k_plane, (float*)v_plane,
                      page_stride, block_table, table_stride, row_slot, row_pos, page_size, q_rank, kv_rank,
                      rot_dim, eps, write_cache, clear_proj), rows);
  if (dtype == LLM_BF16)
    return launched_many_blocks(launch_pdl(latent_store_kernel<bf16>, rows, threads, 0, stream, proj, proj_stride, wq, wc,
                      (const float2*)cos_sin, rot_half, (bf16*)cq_out, (bf16*)k_plane, (bf16*)v_plane,
                      page_stride, block_table, table_stride, row_slot, row_pos, page_size, q_rank, kv_rank,
                      rot_dim, eps, write_cache, clear_proj), rows);
  return LLM_ERR_UNSUPPORTED;
}

LLM_EXPORT int llm_latent_prepare(float* proj, int proj_stride, int q_col, int c_col, const float* wc,
                                  const float* cos_sin, int rot_half, void* q_plain, void* q_full, void* k_plane,
                                  void* v_plane, int dtype, long long page_stride, const int* block_table,
                                  int table_stride, const int* row_slot, const int* row_pos, int rows, int page_size,
                                  int H, int dim, int rot_dim, int kv_rank, float eps, int write_cache, int clear,
                                  cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (H <= 0 || dim < 0 || kv_rank <= 0 || rot_dim < 0 || 2 * rot_half > rot_dim) return LLM_ERR_ARGUMENT;
  if ((long long)H * (dim + rot_dim) >= (1LL << 30)) return LLM_ERR_UNSUPPORTED;
  PrepareArgs a;
  a.proj = proj, a.proj_stride = proj_stride, a.q_col = q_col, a.c_col = c_col, a.wc = wc;
  a.cos_sin = rot_half > 0 ? (const float2*)cos_sin : nullptr, a.rot_half = rot_half, a.page_stride = page_stride;
  a.block_table = block_table, a.row_slot = row_slot, a.row_pos = row_pos, a.table_stride = table_stride;
  a.page_size = page_size, a.H = H, a.dim = dim, a.rot_dim = rot_dim, a.kv_rank = kv_rank, a.eps = eps;
  a.write_cache = write_cache, a.clear = clear;
  const bool vec = ((dim | rot_dim | kv_rank | proj_stride | q_col) & 3) == 0 &&
                   (((uintptr_t)proj | (uintptr_t)q_plain | (uintptr_t)q_full) & 15) == 0;
  // few rows: a piece per thread; many: four, and fewer blocks
  const int pieces = H * (dim + rot_dim) / (vec ? 4 : 1), per = rows >= 512 ? 1024 : 256;
  int shares = (pieces + per - 1) / per;
  shares = shares < 1 ? 1 : shares > 64 ? 64 : shares;
  const dim3 grid(rows, 1 + shares);
  int rc;
#define PREPARE_GO(T)                                                                                           \
  rc = vec ? launch_pdl(latent_prepare_kernel<T, true>, grid, 256, 0, stream, a, (T*)q_plain, (T*)q_full,       \
                        (T*)k_plane, (T*)v_plane)                                                               \
           : launch_pdl(latent_prepare_kernel<T, false>, grid, 256, 0, stream, a, (T*)q_plain, (T*)q_full,      \
                        (T*)k_plane, (T*)v_plane)
  if (dtype == LLM_F32) PREPARE_GO(float);
  else if (dtype == LLM_BF16) PREPARE_GO(bf16);
  else return LLM_ERR_UNSUPPORTED;
#undef PREPARE_GO
  return launched_many_blocks(rc, (long long)rows * (1 + shares));
}

LLM_EXPORT int llm_latent_query(float* q, int q_stride, const float* cos_sin, int rot_half, void* q_plain,
                                void* q_full, int dtype, int rows, int H, int dim, int rot_dim, int kv_rank,
                                int clear, cudaStream_t stream) {
  const long long total = (long long)rows * H * (dim + rot_dim);
  if (total <= 0) return 0;
  if (2 * rot_half > rot_dim) return LLM_ERR_ARGUMENT;
  if ((dim & 3) == 0 && (rot_dim & 3) == 0 && (kv_rank & 3) == 0 && (q_stride & 3) == 0 && total < (1LL << 33) &&
      (((uintptr_t)q | (uintptr_t)q_plain | (uintptr_t)q_full) & 15) == 0) {
    const unsigned pieces = (unsigned)(total >> 2);
    const int vblocks = (int)((pieces + 255) / 256 < 4736 ? (pieces + 255) / 256 : 4736);
    if (dtype == LLM_F32)
      return launched_many_blocks(
          launch_pdl(latent_query_vec_kernel<float>, vblocks, 256, 0, stream, q, q_stride, (const float2*)cos_sin,
                     rot_half, (float*)q_plain, (float*)q_full, pieces, H, dim, rot_dim, kv_rank, clear), vblocks);
    if (dtype == LLM_BF16)
      return launched_many_blocks(
          launch_pdl(latent_query_vec_kernel<bf16>, vblocks, 256, 0, stream, q, q_stride, (const float2*)cos_sin,
                     rot_half, (bf16*)q_plain, (bf16*)q_full, pieces, H, dim, rot_dim, kv_rank, clear), vblocks);
    return LLM_ERR_UNSUPPORTED;
  }
  const int blocks = (int)((total + 255) / 256 < 2368 ? (total + 255) / 256 : 2368);
  if (dtype == LLM_F32)
    return launched_many_blocks(
        launch_pdl(latent_query_kernel<float>, blocks, 256, 0, stream, q, q_stride, (const float2*)cos_sin, rot_half,
                   (float*)q_plain, (float*)q_full, total, H, dim, rot_dim, kv_rank, clear), blocks);
  if (dtype == LLM_BF16)
    return launched_many_blocks(
        launch_pdl(latent_query_kernel<bf16>, blocks, 256, 0, stream, q, q_stride, (const float2*)cos_sin, rot_half,
                   (bf16*)q_plain, (bf16*)q_full, total, H, dim, rot_dim, kv_rank, clear), blocks);
  return LLM_ERR_UNSUPPORTED;
}
