// Heads of attention with two maps over the same values.  With a1 and a2 the two maps' outputs of a
// head (each its own softmax), out = (1 - diff) * unit(a1 - lambda * a2), unit(.) dividing by the
// root mean square over the head's dv channels (eps inside the root).  Everything in 32-bit; rounded
// once.  a [rows][H][2][stride] (dv <= stride: attention may have written whole cache rows), out
// [rows][H][dv].
#include "common.cuh"

namespace {

template <typename T> __device__ __forceinline__ void load8(const T* p, float (&v)[8]);
template <> __device__ __forceinline__ void load8<float>(const float* p, float (&v)[8]) {
  const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
  v[0] = a.x, v[1] = a.y, v[2] = a.z, v[3] = a.w, v[4] = b.x, v[5] = b.y, v[6] = b.z, v[7] = b.w;
}
template <> __device__ __forceinline__ void load8<bf16>(const bf16* p, float (&v)[8]) {
  const uint4 a = *reinterpret_cast<const uint4*>(p);
  const uint32_t w[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) v[2 * i] = __uint_as_float(w[i] << 16), v[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
}
template <typename T> __device__ __forceinline__ void store8(T* p, const float (&v)[8]);
template <> __device__ __forceinline__ void store8<float>(float* p, const float (&v)[8]) {
  reinterpret_cast<float4*>(p)[0] = make_float4(v[0], v[1], v[2], v[3]);
  reinterpret_cast<float4*>(p)[1] = make_float4(v[4], v[5], v[6], v[7]);
}
template <> __device__ __forceinline__ void store8<bf16>(bf16* p, const float (&v)[8]) {
  uint32_t w[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const __nv_bfloat162 t = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
    w[i] = *reinterpret_cast<const uint32_t*>(&t);
  }
  *reinterpret_cast<uint4*>(p) = make_uint4(w[0], w[1], w[2], w[3]);
}

// `lanes` neighbouring threads (a power of two up to 32) share a (row, head); eight channels a
// thread at a time (VEC), or one.
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) two_map_heads_kernel(const T* __restrict__ a, T* __restrict__ out,
                                                            long long items, int dv, int stride, int lanes,
                                                            float lambda, float diff, float eps) {
  constexpr int W = VEC ? 8 : 1;
  pdl_trigger();
  pdl_wait();
  const long long item = ((long long)blockIdx.x * blockDim.x + threadIdx.x) / lanes;
  const int at = threadIdx.x & (lanes - 1);
  const bool have = item < items;
  const T* p1 = a + (size_t)(have ? item : 0) * 2 * stride;
  const T* p2 = p1 + stride;
  float v[W];
  auto read = [&](int c) {
    if constexpr (VEC) {
      float x[8], y[8];
      load8<T>(p1 + c, x), load8<T>(p2 + c, y);
#pragma unroll
      for (int i = 0; i < 8; ++i) v[i] = fmaf(-lambda, y[i], x[i]);
    } else {
      v[0] = fmaf(-lambda, to_f32(p2[c]), to_f32(p1[c]));
    }
  };
  float ss = 0.f;
  for (int c = at * W; c < dv; c += lanes * W) {
    read(c);
#pragma unroll
    for (int i = 0; i < W; ++i) ss = fmaf(v[i], v[i], ss);
  }
  for (int o = lanes >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  if (!have) return;
  const float scale = (1.f - diff) / sqrtf(ss / (float)dv + eps);
  T* dst = out + (size_t)item * dv;
  const bool once = dv <= lanes * W;      // what was read is still in registers
  for (int c = at * W; c < dv; c += lanes * W) {
    if (!once) read(c);
#pragma unroll
    for (int i = 0; i < W; ++i) v[i] *= scale;
    if constexpr (VEC) store8<T>(dst + c, v);
    else dst[c] = from_f32<T>(v[0]);
  }
}

template <typename T>
int launch_two_map_heads(const T* a, T* out, int rows, int H, int dv, int stride, float lambda, float diff, float eps,
                         cudaStream_t stream) {
  const bool vec = dv % 8 == 0 && stride % 8 == 0 && (((uintptr_t)a | (uintptr_t)out) & 15) == 0;
  const int pieces = vec ? dv / 8 : dv;
  int lanes = 1;
  while (lanes < 32 && lanes < pieces) lanes *= 2;
  const long long items = (long long)rows * H;
  const long long blocks = (items * lanes + 255) / 256;
  if (blocks > 0x7fffffffLL) return LLM_ERR_UNSUPPORTED;
  const int rc = vec ? launch_pdl(two_map_heads_kernel<T, true>, (unsigned)blocks, 256, 0, stream, a, out, items, dv,
                                  stride, lanes, lambda, diff, eps)
                     : launch_pdl(two_map_heads_kernel<T, false>, (unsigned)blocks, 256, 0, stream, a, out, items, dv,
                                  stride, lanes, lambda, diff, eps);
  // (it stands in front of the output projection: see launched_many_blocks)
  return launched_many_blocks(rc, blocks);
}
}  // namespace

LLM_EXPORT int llm_two_map_heads(const void* a, void* out, int dtype, int rows, int H, int dv, int stride,
                                 float lambda, float diff, float eps, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (H <= 0 || dv <= 0 || stride < dv) return LLM_ERR_ARGUMENT;
  if (dtype == LLM_F32)
    return launch_two_map_heads<float>((const float*)a, (float*)out, rows, H, dv, stride, lambda, diff, eps, stream);
  if (dtype == LLM_BF16)
    return launch_two_map_heads<bf16>((const bf16*)a, (bf16*)out, rows, H, dv, stride, lambda, diff, eps, stream);
  return LLM_ERR_UNSUPPORTED;
}
