// Per-head preparation of projected rows before attention: an optional weighted RMS norm over the head, rotary positions on a
// run of its dimensions, and the move to where the attention reads it -- in place, to a dense buffer, or scattered into the
// rows of a cache.
//
//   z = head / sqrt(mean(head^2) + eps) * w                    (optional; statistics over the whole head, fp32 -- or, norm_all, over all
//                                                              heads of the group at once, with one weight per number of the group)
//   (u, v) <- (u cos a - v sin a, v cos a + u sin a) * mag     for the pairs of dimensions [rot_off, rot_off + rot_dims):
//             pair i = (2 i, 2 i + 1) when interleaved, else (i, i + rot_dims / 2); a = position * freq[i] in fp32, or with fp64
//             frequencies in fp64 and reduced to [-pi, pi] before the fp32 sine and cosine
//   the other dimensions pass unchanged.
//
// Up to four groups of heads (e.g. the queries and keys of two mixers that share one fused projection) run as one launch; one CTA per (row,
// group).  A group may be written in fp32 whatever the dtype it is read in (operands of an fp32 recurrence).
#include "common.cuh"

namespace b200 {

namespace {

constexpr int kHrThreads = 128, kHrMaxSegs = 4;

struct HeadSeg {
  const void* in; void* out; const void* norm_w; const void* freq; const int64_t* out_rows;
  int64_t ld_in, ld_out;
  int heads, dim, in_stride, out_stride, rot_off, rot_dims, interleaved;
  float mag;
  int norm_all, freq_f64, out_f32;
};
struct HeadSegs { HeadSeg s[kHrMaxSegs]; };

// grid (rows, groups): the CTA of a row works out the row's cosines and sines once (they depend on the position and the pair only, not
// on the head), then its warps take the heads of the group in turn
template <typename T, typename TO>
__device__ __forceinline__ void head_rope_row(const HeadSeg& s, const int* __restrict__ row_pos, float eps) {
  extern __shared__ __align__(16) float hr_smem[];   // [rot_dims / 2] cosines, then as many sines, both times mag
  __shared__ float s_part[kHrThreads / 32];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int64_t row = blockIdx.x;
  const int64_t orow = s.out_rows ? s.out_rows[row] : row;
  if (orow < 0) return;   // a row with nowhere to go (the whole CTA leaves: no barrier is left waiting)
  const int half = s.rot_dims / 2;
  float* const cs = hr_smem;
  float* const sn = hr_smem + half;
  if (half > 0) {
    const int pos = row_pos[row];
    for (int i = threadIdx.x; i < half; i += kHrThreads) {
      float ang, a, b;
      if (s.freq_f64) {
        double t = (double)pos * reinterpret_cast<const double*>(s.freq)[i];
        t -= 6.283185307179586476925286766559 * rint(t * 0.15915494309189533576888376337251);
        ang = (float)t;
      } else {
        ang = (float)pos * reinterpret_cast<const float*>(s.freq)[i];
      }
      sincosf(ang, &a, &b);
      sn[i] = a * s.mag;
      cs[i] = b * s.mag;
    }
    __syncthreads();
  }
  const T* wall = reinterpret_cast<const T*>(s.norm_w);
  float rstd_all = 1.0f;
  if (s.norm_all) {   // every number of the row is read before the first is written: the barrier of the sum stands between
    const T* x = reinterpret_cast<const T*>(s.in) + row * s.ld_in;
    const int n = s.heads * s.dim;   // the heads lie side by side
    float ss = 0.f;
    if (vec8_ok(n, x)) {
      for (int i = threadIdx.x * 8; i < n; i += kHrThreads * 8) {
        float v[8];
        load8(x + i, v);
#pragma unroll
        for (int j = 0; j < 8; ++j) ss = fmaf(v[j], v[j], ss);
      }
    } else {
      for (int i = threadIdx.x; i < n; i += kHrThreads) { const float v = load_as_float(x, i); ss = fmaf(v, v, ss); }
    }
    ss = warp_sum(ss);
    if (lane == 0) s_part[warp] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < kHrThreads / 32; ++i) ss += s_part[i];
    rstd_all = 1.0f / sqrtf(ss / (float)n + eps);
  }
  for (int h = warp; h < s.heads; h += kHrThreads / 32) {
    const T* x = reinterpret_cast<const T*>(s.in) + row * s.ld_in + (int64_t)h * s.in_stride;
    TO* o = reinterpret_cast<TO*>(s.out) + orow * s.ld_out + (int64_t)h * s.out_stride;
    const T* w = s.norm_all ? wall + (int64_t)h * s.dim : wall;
    float rstd = rstd_all;
    if (w && !s.norm_all) {
      float ss = 0.f;
      for (int i = lane; i < s.dim; i += 32) { const float v = load_as_float(x, i); ss = fmaf(v, v, ss); }
      rstd = 1.0f / sqrtf(warp_sum(ss) / (float)s.dim + eps);   // the shuffle also orders every lane's reads before any write below
    }
    // the rotated pairs: both members are read before either is written, and no other lane touches them
    for (int i = lane; i < half; i += 32) {
      const int a = s.rot_off + (s.interleaved ? 2 * i : i), b = s.rot_off + (s.interleaved ? 2 * i + 1 : i + half);
      float u = load_as_float(x, a), v = load_as_float(x, b);
      if (w) { u = u * rstd * load_as_float(w, a); v = v * rstd * load_as_float(w, b); }
      store_from_float(o, a, u * cs[i] - v * sn[i]);
      store_from_float(o, b, v * cs[i] + u * sn[i]);
    }
    const bool moved = (const void*)o != (const void*)x;
    if (!w && !moved) continue;
    for (int i = lane; i < s.dim; i += 32) {
      if (i >= s.rot_off && i < s.rot_off + 2 * half) continue;
      float v = load_as_float(x, i);
      if (w) v = v * rstd * load_as_float(w, i);
      store_from_float(o, i, v);
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(kHrThreads) head_rope_kernel(HeadSegs S, const int* __restrict__ row_pos, float eps) {
  griddep_launch();
  griddep_wait();
  const HeadSeg s = S.s[blockIdx.y];
  if (s.out_f32) head_rope_row<T, float>(s, row_pos, eps);
  else head_rope_row<T, T>(s, row_pos, eps);
}

}  // namespace

}  // namespace b200

using namespace b200;

extern "C" {

int b200_head_rope(const b200_head_rope_seg* segs, int n_segs, const int32_t* row_pos, int64_t rows, float eps, int dtype, b200_stream_t stream) {
  B200_CHECK_ARG(segs && n_segs >= 1 && n_segs <= kHrMaxSegs && row_pos, "b200_head_rope: one to four groups of heads and the rows' positions");
  B200_CHECK_ARG(rows > 0 && rows <= 0x7fffffff, "b200_head_rope: bad row count");
  HeadSegs S;
  int max_rot = 0;
  for (int i = 0; i < kHrMaxSegs; ++i) {
    const b200_head_rope_seg& a = segs[i < n_segs ? i : 0];
    B200_CHECK_ARG(a.in && a.out && a.heads > 0 && a.dim > 0, "b200_head_rope: null pointer or empty head");
    B200_CHECK_ARG(a.rot_dims >= 0 && a.rot_dims % 2 == 0 && a.rot_off >= 0 && a.rot_off + a.rot_dims <= a.dim && (a.rot_dims == 0 || a.freq),
                   "b200_head_rope: the rotated dimensions must be an even run inside the head, with their frequencies");
    B200_CHECK_ARG(!a.norm_all || (a.norm_w && (a.in_stride == a.dim || a.heads == 1)), "b200_head_rope: a norm over all heads needs its weight and heads side by side");
    S.s[i] = HeadSeg{a.in, a.out, a.norm_w, a.freq, a.out_rows, a.ld_in, a.ld_out, a.heads, a.dim, a.in_stride, a.out_stride, a.rot_off, a.rot_dims,
                     a.interleaved, a.mag, a.norm_all, a.freq_f64, a.out_f32};
    if (i < n_segs) max_rot = a.rot_dims > max_rot ? a.rot_dims : max_rot;
  }
  B200_CHECK_ARG(max_rot <= 8192, "b200_head_rope: at most 8192 rotated dimensions");
  B200_FLOAT_TYPES(dtype, T, B200_CUDA(launch(head_rope_kernel<T>, dim3((unsigned)rows, (unsigned)n_segs), dim3(kHrThreads), (size_t)max_rot * sizeof(float),
                                               (cudaStream_t)stream, S, row_pos, eps)));
  return B200_OK;
}

}  // extern "C"
