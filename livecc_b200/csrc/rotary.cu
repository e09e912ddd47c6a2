// Rotary positions in the rotate-half layout on slices of a projection, written as fp32 for a recurrence that keeps
// its operands in fp32. Positions, angles, cos and sin are fp32 (full-range sinf / cosf, no fast-math).
#include <math.h>

#include "common.cuh"
#include "launch.h"
#include "seqmix.h"

namespace lcc {
namespace {

template <typename T> __device__ __forceinline__ float ldf(const T* p);
template <> __device__ __forceinline__ float ldf<float>(const float* p) { return *p; }
template <> __device__ __forceinline__ float ldf<bf16>(const bf16* p) { return __bfloat162float(*p); }

__device__ __forceinline__ void ld4(const float* p, float (&v)[4]) {
    const float4 u = *reinterpret_cast<const float4*>(p);
    v[0] = u.x; v[1] = u.y; v[2] = u.z; v[3] = u.w;
}
__device__ __forceinline__ void ld4(const bf16* p, float (&v)[4]) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y);
    v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
}

__device__ __forceinline__ int seq_past(const SeqPos& p) { return p.kv_len ? *p.kv_len : p.past; }
__device__ __forceinline__ bool seq_done(const SeqPos& p) { return p.finished && *p.finished; }

struct Segs { RotarySegment s[4]; int n; };

// gridDim.y CTAs per row (several when the call has few rows, so that a decode step's single row is not one CTA's serial
// walk); together their threads walk the output channels of every segment.
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) rotary_pack_kernel(const T* __restrict__ in, int ld_in, float* __restrict__ out, int ld_out,
                                                          Segs segs, const float* __restrict__ inv_freq, float mag,
                                                          const float* __restrict__ fill, float* __restrict__ fill_out, int fill_n,
                                                          SeqPos pos) {
    if (seq_done(pos)) return;
    const int t = blockIdx.x;
    const float p = (float)(seq_past(pos) + t);
    const T* row = in + (size_t)t * ld_in;
    float* orow = out + (size_t)t * ld_out;
    for (int si = 0; si < segs.n; ++si) {
        const RotarySegment sg = segs.s[si];
        const int n = sg.heads * sg.dim, half = sg.rot_dims / 2;
        if (VEC && sg.rot_dims == 0) {       // nothing turns: four neighbouring channels per thread
            for (int i = (threadIdx.x + blockIdx.y * blockDim.x) * 4; i < n; i += blockDim.x * gridDim.y * 4) {
                float v[4];
                ld4(row + sg.col_in + i, v);
#pragma unroll
                for (int u = 0; u < 4; ++u) v[u] = (sg.silu ? v[u] / (1.f + expf(-v[u])) : v[u]) * sg.scale;
                *reinterpret_cast<float4*>(orow + sg.col_out + i) = make_float4(v[0], v[1], v[2], v[3]);
            }
            continue;
        }
        for (int i = threadIdx.x + blockIdx.y * blockDim.x; i < n; i += blockDim.x * gridDim.y) {
            const int d = i % sg.dim, hb = i - d;
            const int r = d - sg.rot_off;
            float v = ldf(row + sg.col_in + i);
            if (sg.silu) v = v / (1.f + expf(-v));
            if (r >= 0 && r < sg.rot_dims) {
                const int j = r < half ? r : r - half;
                const float ang = p * inv_freq[j];
                const float c = cosf(ang) * mag, s = sinf(ang) * mag;
                float other = ldf(row + sg.col_in + hb + sg.rot_off + (r < half ? r + half : r - half));
                if (sg.silu) other = other / (1.f + expf(-other));
                v = r < half ? v * c - other * s : v * c + other * s;
            }
            orow[sg.col_out + i] = v * sg.scale;
        }
    }
    if (fill_out && blockIdx.y == 0)
        for (int i = threadIdx.x; i < fill_n; i += blockDim.x) fill_out[(size_t)t * fill_n + i] = fill[i];
}

}  // namespace

int rotary_pack_f32(int dt, const void* in, int ld_in, float* out, int ld_out, const RotarySegment* seg, int n_seg,
                    const float* inv_freq, float mag, const float* fill, float* fill_out, int fill_n, int S, SeqPos pos,
                    cudaStream_t s) {
    if (!in || !out || !seg || n_seg < 1 || n_seg > 4 || S < 1 || (fill_out && (!fill || fill_n < 1))) return -2;
    Segs g{};
    g.n = n_seg;
    for (int i = 0; i < n_seg; ++i) {
        g.s[i] = seg[i];
        if (seg[i].rot_dims < 0 || (seg[i].rot_dims & 1) || seg[i].rot_off < 0 || seg[i].rot_off + seg[i].rot_dims > seg[i].dim ||
            (seg[i].rot_dims > 0 && !inv_freq))
            return -2;
    }
    count_launch();
    const dim3 S_grid(S, S < 32 ? 8 : 1);
    // four channels per thread in segments without a rotation, when every row and segment starts on a whole group
    bool vec = (ld_in % 4) == 0 && (ld_out % 4) == 0 && ((uintptr_t)in % (4 * dt_size(dt))) == 0 && ((uintptr_t)out % 16) == 0;
    bool any = false;
    for (int i = 0; i < n_seg; ++i) {
        vec = vec && (seg[i].col_in % 4) == 0 && (seg[i].col_out % 4) == 0 && (seg[i].heads * seg[i].dim) % 4 == 0;
        any = any || seg[i].rot_dims == 0;
    }
    vec = vec && any;
#define LCC_PACK(T, V) rotary_pack_kernel<T, V><<<S_grid, 256, 0, s>>>((const T*)in, ld_in, out, ld_out, g, inv_freq, mag, fill, fill_out, fill_n, pos)
    if (dt == DT_F32) { if (vec) LCC_PACK(float, true); else LCC_PACK(float, false); }
    else { if (vec) LCC_PACK(bf16, true); else LCC_PACK(bf16, false); }
#undef LCC_PACK
    return cudaGetLastError() == cudaSuccess ? 0 : -100;
}

}  // namespace lcc
