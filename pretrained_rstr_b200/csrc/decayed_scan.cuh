// Core of a linear recurrence over a matrix state with decays, shared by the mixers that have
// one (decayed_scan.cu, state_space.cu).  Per head, with keys k and queries q of `dim` numbers,
// values v of `vdim` and a decay a in (0, 1] per key channel or per head,
//
//     S_t = diag(a_t) S_(t-1) + k_t v_t^T              o_t = S_t^T q_t
//
// The state lies as [vdim][dim].  A thread holds KPL neighbouring keys of CC value columns (4 or 8)
// in registers; the `dim` keys of a column are spread over L neighbouring lanes (a power of two
// from 8 to 32).  A decay travels as c = a - 1 and a step is S + (k v + c S), so that a decay
// close to one keeps its precision.  The order of every sum depends on the sizes only.
#pragma once
#include "common.cuh"

namespace dscan {
inline int keys_per_lane(int dim) { return dim <= 128 ? 4 : dim <= 256 ? 8 : 16; }
// Lanes a column is spread over (0: beyond the kernels).
inline int lanes_of(int dim) {
    if (dim <= 0 || dim > 512) return 0;
    const int kpl = keys_per_lane(dim);
    int lanes = 8;
    while (lanes * kpl < dim) lanes *= 2;
    return lanes;
}

// The numbers of a thread's columns c0 .. c0 + CC - 1 from or to rows of `dim` numbers.
template <int CC, int KPL>
__device__ __forceinline__ void load_state(float (&S)[CC][KPL], const float* from, int ln, int c0,
                                           int dim, int vdim) {
    const bool vec = dim % 4 == 0;
#pragma unroll
    for (int c = 0; c < CC; ++c) {
        const bool live = from != nullptr && c0 + c < vdim;
        const float* row = from + (size_t)(c0 + c) * dim;
        if (vec) {
#pragma unroll
            for (int g = 0; g < KPL / 4; ++g) {
                const int kk = ln * KPL + 4 * g;
                const float4 x = live && kk < dim ? *reinterpret_cast<const float4*>(row + kk)
                                                  : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                S[c][4 * g] = x.x; S[c][4 * g + 1] = x.y; S[c][4 * g + 2] = x.z; S[c][4 * g + 3] = x.w;
            }
        } else {
#pragma unroll
            for (int i = 0; i < KPL; ++i) {
                const int kk = ln * KPL + i;
                S[c][i] = live && kk < dim ? row[kk] : 0.0f;
            }
        }
    }
}
template <int CC, int KPL>
__device__ __forceinline__ void store_state(const float (&S)[CC][KPL], float* to, int ln, int c0,
                                            int dim, int vdim) {
    const bool vec = dim % 4 == 0;
#pragma unroll
    for (int c = 0; c < CC; ++c) {
        if (c0 + c >= vdim) continue;
        float* row = to + (size_t)(c0 + c) * dim;
        if (vec) {
#pragma unroll
            for (int g = 0; g < KPL / 4; ++g) {
                const int kk = ln * KPL + 4 * g;
                if (kk < dim)
                    *reinterpret_cast<float4*>(row + kk) =
                        make_float4(S[c][4 * g], S[c][4 * g + 1], S[c][4 * g + 2], S[c][4 * g + 3]);
            }
        } else {
#pragma unroll
            for (int i = 0; i < KPL; ++i) {
                const int kk = ln * KPL + i;
                if (kk < dim) row[kk] = S[c][i];
            }
        }
    }
}

// One token: k, c, q point at the lane's KPL numbers (c at one number when !PER_KEY), v holds the
// thread's values (already times the key's scale).  part[c] = the lane's share of q . S.
template <int CC, int KPL, bool PER_KEY, bool OUT>
__device__ __forceinline__ void advance(float (&S)[CC][KPL], const float* k, const float* c, const float* q,
                                        const float (&v)[CC], float (&part)[CC]) {
    const float c1 = PER_KEY ? 0.0f : c[0];
#pragma unroll
    for (int j = 0; j < CC; ++j) part[j] = 0.0f;
#pragma unroll
    for (int g = 0; g < KPL / 4; ++g) {
        const float4 k4 = reinterpret_cast<const float4*>(k)[g];
        const float4 c4 = PER_KEY ? reinterpret_cast<const float4*>(c)[g] : make_float4(c1, c1, c1, c1);
        const float4 q4 = OUT ? reinterpret_cast<const float4*>(q)[g] : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
        for (int j = 0; j < CC; ++j) {
            float* s = &S[j][4 * g];
            s[0] += fmaf(c4.x, s[0], k4.x * v[j]);
            s[1] += fmaf(c4.y, s[1], k4.y * v[j]);
            s[2] += fmaf(c4.z, s[2], k4.z * v[j]);
            s[3] += fmaf(c4.w, s[3], k4.w * v[j]);
            if (OUT) {
                part[j] = fmaf(s[0], q4.x, part[j]);
                part[j] = fmaf(s[1], q4.y, part[j]);
                part[j] = fmaf(s[2], q4.z, part[j]);
                part[j] = fmaf(s[3], q4.w, part[j]);
            }
        }
    }
}

// Sums of the lanes' CC shares: halves of the columns change sides until a lane holds one, which the
// lanes left over close.  Afterwards lane ln holds column held_column(ln, L), and the lanes with
// (ln & (L / CC - 1)) == 0 cover them all.
template <int CC>
__device__ __forceinline__ float close_columns(const float (&p)[CC], int ln, int L) {
    float a[CC];
#pragma unroll
    for (int j = 0; j < CC; ++j) a[j] = p[j];
    int h = L >> 1;
#pragma unroll
    for (int n = CC / 2; n > 0; n >>= 1, h >>= 1) {
        const bool up = (ln & h) != 0;
#pragma unroll
        for (int j = 0; j < n; ++j) {
            const float keep = up ? a[n + j] : a[j], send = up ? a[j] : a[n + j];
            a[j] = keep + __shfl_xor_sync(0xffffffffu, send, h);
        }
    }
    for (; h > 0; h >>= 1) a[0] += __shfl_xor_sync(0xffffffffu, a[0], h);
    return a[0];
}
template <int CC>
__device__ __forceinline__ int held_column(int ln, int L) {
    int j = 0;
#pragma unroll
    for (int n = CC / 2, h = L >> 1; n > 0; n >>= 1, h >>= 1) j += (ln & h) ? n : 0;
    return j;
}

__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }
// T: the type the result is stored in; one that keeps 8 bits of mantissa is content with the
// hardware's exponential.
template <typename T>
__device__ __forceinline__ float silu(float z) {
    return __fdividef(z, 1.0f + (sizeof(T) == 2 ? __expf(-z) : expf(-z)));
}

// Portions in segments of DS_SEG tokens; segment z of the launch is segment s of request b
// (requests' segments are numbered in request order).
constexpr int DS_SEG = 64;
__device__ __forceinline__ bool find_segment(const int* q_start, int n_requests, int z, int& b, int& s,
                                             int& nseg) {
    int base = 0;
    for (b = 0; b < n_requests; ++b) {
        const int n = q_start[b + 1] - q_start[b];
        nseg = n > 0 ? (n + DS_SEG - 1) / DS_SEG : 0;
        if (z < base + nseg) {
            s = z - base;
            return true;
        }
        base += nseg;
    }
    return false;
}

__device__ __forceinline__ void copy16(void* smem, const void* gmem) {
    const unsigned d = (unsigned)__cvta_generic_to_shared(smem);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d), "l"(gmem) : "memory");
}
__device__ __forceinline__ void copy_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void copy_wait() {
    asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}
}  // namespace dscan
