// Activations between the two products of a feed-forward, a launch each:
//
// expert_act: a router that scores by the softmax over all experts and chooses by score plus a
//   correction per expert, and the gated activation of the chosen experts with their weights (the
//   scores without the correction, optionally shares of their sum, times a constant).  The last
//   `identity` of the router's experts give back the feed-forward's input: their weight times the
//   input joins the stream here.  An optional shared expert runs for every token, optionally times
//   sigmoid of one more column.
// act_columns: act(in) of a range of columns.
// Inputs are columns of one 32-bit product; results in the products' type.  32-bit arithmetic.
#include "common.cuh"

namespace {
__device__ __forceinline__ float ea_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
// 0: silu, 1: gelu (tanh form).  O: the type the result is stored in; one that keeps 8 bits of
// mantissa is content with the hardware's exponential.
template <typename O>
__device__ __forceinline__ float ea_gate(float g, int act) {
    if (act == 1) return prb_activate(g, PRB_ACT_GELU_TANH);
    return __fdividef(g, 1.0f + (sizeof(O) == 2 ? __expf(-g) : expf(-g)));
}

// Floats in an order that unsigned integers keep (for the warp's integer reductions).
__device__ __forceinline__ unsigned ordered(float v) {
    const unsigned b = __float_as_uint(v);
    return (b & 0x80000000u) ? ~b : b | 0x80000000u;
}
__device__ __forceinline__ float from_ordered(unsigned k) {
    return __uint_as_float((k & 0x80000000u) ? k & 0x7fffffffu : ~k);
}

struct ExpertArgs {
    void* out; long out_ld;
    const float* in; long in_ld;
    int gate_col, up_col, router_col, shared_gate_col, shared_up_col, shared_weight_col;
    int n_rows, experts, identity, top, group, shared, renorm, act;
    float factor;
    const float* correction;         // [experts + identity], or null
    // identity experts: x += weight * h, with h given or (h == null) x / rms(x) * norm_w
    float* x; long x_ld; int width;
    const void* h; long h_ld;
    const float* norm_w;
    float eps;
};

// Scores, choice and weights of one row, by a warp: wt[e] of every expert, own[0] the identity experts'
// weight together, own[1] the shared expert's.
__device__ __forceinline__ void choose(const ExpertArgs& a, const float* row, float* sc, float* pick, float* wt,
                                       float* own) {
    const int lane = threadIdx.x & 31, all = a.experts + a.identity;
    float top_z = -INFINITY;
    for (int e = lane; e < all; e += 32) {
        const float z = row[a.router_col + e];
        sc[e] = z;
        top_z = fmaxf(top_z, z);
    }
    top_z = from_ordered(__reduce_max_sync(0xffffffffu, ordered(top_z)));
    float sum = 0.0f;
    for (int e = lane; e < all; e += 32) {
        const float p = expf(sc[e] - top_z);
        sc[e] = p;
        sum += p;
    }
    sum = prb_warp_sum(sum);
    for (int e = lane; e < all; e += 32) {
        const float s = sc[e] / sum;
        sc[e] = s;
        pick[e] = s + (a.correction ? a.correction[e] : 0.0f);
        wt[e] = 0.0f;
    }
    __syncwarp();
    float chosen = 0.0f;
    for (int k = 0; k < a.top; ++k) {                // the largest left; ties: the lower index
        float best = -INFINITY;
        unsigned arg = all;
        for (int e = lane; e < all; e += 32) {
            const float v = pick[e];
            if (v > best) { best = v; arg = e; }
        }
        const unsigned key = ordered(best);
        const unsigned top_key = __reduce_max_sync(0xffffffffu, key);
        arg = __reduce_min_sync(0xffffffffu, key == top_key ? arg : (unsigned)all);
        if (arg >= all) break;                       // (a row of NaNs: padding, or a fault upstream)
        chosen += sc[arg];
        if (lane == 0) {
            wt[arg] = sc[arg];
            pick[arg] = -INFINITY;
        }
        __syncwarp();
    }
    const float mult = a.factor / (a.renorm ? chosen : 1.0f);
    float mine = 0.0f;
    for (int e = lane; e < all; e += 32) {
        const float w = wt[e] * mult;
        wt[e] = w;
        if (e >= a.experts) mine += w;
    }
    mine = prb_warp_sum(mine);
    if (lane == 0) {
        own[0] = mine;
        own[1] = a.shared_weight_col >= 0 ? ea_sigmoid(row[a.shared_weight_col]) : 1.0f;
    }
}

struct Columns {
    int n_exp, n_all, lo, hi;        // the routed experts' columns, all, and this CTA's slice
    bool vec;
    __device__ __forceinline__ explicit Columns(const ExpertArgs& a, int esz) {
        n_exp = a.experts * a.group;
        n_all = n_exp + a.shared;
        const int per = ((n_all + (int)gridDim.y - 1) / (int)gridDim.y + 3) / 4 * 4;
        lo = blockIdx.y * per;
        hi = min(n_all, lo + per);
        vec = a.group % 4 == 0 && (a.gate_col | a.up_col | a.in_ld | a.out_ld) % 4 == 0 &&
              (a.shared == 0 || (a.shared_gate_col | a.shared_up_col | a.shared) % 4 == 0) &&
              ((uintptr_t)a.in) % 16 == 0 && ((uintptr_t)a.out) % (4 * esz) == 0;
    }
    __device__ __forceinline__ int gate(const ExpertArgs& a, int i) const {
        return i < n_exp ? a.gate_col + i : a.shared_gate_col + i - n_exp;
    }
    __device__ __forceinline__ int up(const ExpertArgs& a, int i) const {
        return i < n_exp ? a.up_col + i : a.shared_up_col + i - n_exp;
    }
};

// Few rows: CTAs (row, slice of its columns); every CTA of a row chooses for itself.  Columns are
// the experts' (experts * group), then the shared expert's.
template <typename O>
__global__ void __launch_bounds__(256) expert_act_row_kernel(ExpertArgs a) {
    extern __shared__ float sh[];                    // [all] scores, [all] choice, [all] weights
    __shared__ float scratch[32];
    __shared__ float own_s[2];
    const int all = a.experts + a.identity, t = blockIdx.x;
    prb_grid_launch_dependents();
    const Columns c(a, sizeof(O));
    const float* row = a.in + (size_t)t * a.in_ld;
    const float* wt = sh + 2 * all;
    prb_grid_wait();
    // the first columns are asked for before anyone knows which experts the row chooses
    const int first = c.lo + (int)threadIdx.x * 4;
    float4 g0 = make_float4(0.0f, 0.0f, 0.0f, 0.0f), u0 = g0;
    if (c.vec && first < c.hi) {
        g0 = *reinterpret_cast<const float4*>(row + c.gate(a, first));
        u0 = *reinterpret_cast<const float4*>(row + c.up(a, first));
    }
    if (threadIdx.x < 32) choose(a, row, sh, sh + all, sh + 2 * all, own_s);
    __syncthreads();
    O* o = (O*)a.out + (size_t)t * a.out_ld;
    if (c.vec) {
        for (int i = first; i < c.hi; i += blockDim.x * 4) {
            const float w = i < c.n_exp ? wt[i / a.group] : own_s[1];
            float v[4] = {0.0f, 0.0f, 0.0f, 0.0f};
            if (w != 0.0f) {                         // (columns of experts not chosen are not read)
                float4 g = g0, u = u0;
                if (i != first) {
                    g = *reinterpret_cast<const float4*>(row + c.gate(a, i));
                    u = *reinterpret_cast<const float4*>(row + c.up(a, i));
                }
                v[0] = w * ea_gate<O>(g.x, a.act) * u.x;
                v[1] = w * ea_gate<O>(g.y, a.act) * u.y;
                v[2] = w * ea_gate<O>(g.z, a.act) * u.z;
                v[3] = w * ea_gate<O>(g.w, a.act) * u.w;
            }
            prb_store4(o + i, v[0], v[1], v[2], v[3]);
        }
    } else {
        for (int i = c.lo + threadIdx.x; i < c.hi; i += blockDim.x) {
            const float w = i < c.n_exp ? wt[i / a.group] : own_s[1];
            o[i] = prb_from_float<O>(w != 0.0f ? w * ea_gate<O>(row[c.gate(a, i)], a.act) * row[c.up(a, i)] : 0.0f);
        }
    }
    if (a.identity == 0 || blockIdx.y != 0 || own_s[0] == 0.0f) return;
    float* x = a.x + (size_t)t * a.x_ld;
    if (a.h != nullptr) {
        const O* h = (const O*)a.h + (size_t)t * a.h_ld;
        for (int i = threadIdx.x; i < a.width; i += blockDim.x)
            x[i] = fmaf(own_s[0], prb_to_float<O>(h[i]), x[i]);
        return;
    }
    float ss = 0.0f;
    for (int i = threadIdx.x; i < a.width; i += blockDim.x) ss = fmaf(x[i], x[i], ss);
    ss = prb_block_sum(ss, scratch);
    const float inv = own_s[0] / sqrtf(ss / (float)a.width + a.eps);
    for (int i = threadIdx.x; i < a.width; i += blockDim.x)
        x[i] = fmaf(x[i] * inv, a.norm_w ? a.norm_w[i] : 1.0f, x[i]);
}

// `n` columns of a row by a warp: w * f(gate) * up, or zeros without reading anything.
template <typename O>
__device__ __forceinline__ void act_run(O* __restrict__ o, const float* __restrict__ gate,
                                        const float* __restrict__ up, int n, float w, int act, bool vec, int lane) {
    if (vec) {
        if (w == 0.0f) {
            for (int i = lane * 4; i < n; i += 128) prb_store4(o + i, 0.0f, 0.0f, 0.0f, 0.0f);
            return;
        }
#pragma unroll 4
        for (int i = lane * 4; i < n; i += 128) {
            const float4 g = *reinterpret_cast<const float4*>(gate + i);
            const float4 u = *reinterpret_cast<const float4*>(up + i);
            prb_store4(o + i, w * ea_gate<O>(g.x, act) * u.x, w * ea_gate<O>(g.y, act) * u.y, w * ea_gate<O>(g.z, act) * u.z,
                       w * ea_gate<O>(g.w, act) * u.w);
        }
        return;
    }
    for (int i = lane; i < n; i += 32)
        o[i] = prb_from_float<O>(w != 0.0f ? w * ea_gate<O>(gate[i], act) * up[i] : 0.0f);
}

// Many rows: a warp a row and slice, no barrier.  A slice is every gridDim.y-th expert, the shared
// expert (in shares) and a share of the identity experts' width.
constexpr int EA_ROWS = 8;
template <typename O>
__global__ void __launch_bounds__(EA_ROWS * 32) expert_act_kernel(ExpertArgs a) {
    extern __shared__ float sh[];                    // per row: [all] scores, [all] choice, [all] weights
    __shared__ float own_s[EA_ROWS][2];
    const int all = a.experts + a.identity, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    prb_grid_launch_dependents();
    const int t = blockIdx.x * EA_ROWS + warp;
    if (t >= a.n_rows) return;
    const bool vec = Columns(a, sizeof(O)).vec;
    const float* row = a.in + (size_t)t * a.in_ld;
    float* mine = sh + (size_t)warp * 3 * all;
    const float* wt = mine + 2 * all;
    choose(a, row, mine, mine + all, mine + 2 * all, own_s[warp]);
    __syncwarp();
    const float identity = own_s[warp][0], shared_w = own_s[warp][1];
    O* o = (O*)a.out + (size_t)t * a.out_ld;
    for (int e = blockIdx.y; e < a.experts; e += gridDim.y)
        act_run<O>(o + (size_t)e * a.group, row + a.gate_col + (size_t)e * a.group,
                   row + a.up_col + (size_t)e * a.group, a.group, wt[e], a.act, vec, lane);
    if (a.shared > 0) {
        const int per = ((a.shared + (int)gridDim.y - 1) / (int)gridDim.y + 3) / 4 * 4;
        const int lo = blockIdx.y * per, n = min(a.shared - lo, per);
        if (n > 0)
            act_run<O>(o + (size_t)a.experts * a.group + lo, row + a.shared_gate_col + lo,
                       row + a.shared_up_col + lo, n, shared_w, a.act, vec, lane);
    }
    if (a.identity == 0 || identity == 0.0f) return;
    float* x = a.x + (size_t)t * a.x_ld;
    if (a.h != nullptr) {                            // (every slice a share of the width)
        const O* h = (const O*)a.h + (size_t)t * a.h_ld;
        const int per = ((a.width + (int)gridDim.y - 1) / (int)gridDim.y + 127) / 128 * 128;
        const int end = min(a.width, ((int)blockIdx.y + 1) * per);
        for (int i0 = blockIdx.y * per + lane; i0 < end; i0 += 128) {
            float xv[4], hv[4];
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                const int i = i0 + 32 * k;
                xv[k] = i < end ? x[i] : 0.0f;
                hv[k] = i < end ? prb_to_float<O>(h[i]) : 0.0f;
            }
#pragma unroll
            for (int k = 0; k < 4; ++k)
                if (i0 + 32 * k < end) x[i0 + 32 * k] = fmaf(identity, hv[k], xv[k]);
        }
        return;
    }
    if (blockIdx.y != 0) return;
    float ss = 0.0f;
    for (int i = lane; i < a.width; i += 32) ss = fmaf(x[i], x[i], ss);
    const float inv = identity / sqrtf(prb_warp_sum(ss) / (float)a.width + a.eps);
    for (int i = lane; i < a.width; i += 32) x[i] = fmaf(x[i] * inv, a.norm_w ? a.norm_w[i] : 1.0f, x[i]);
}

__device__ __forceinline__ float column_act(float v, int act) {
    switch (act) {
        case 0: { const float r = fmaxf(v, 0.0f); return r * r; }
        case 1: return fmaxf(v, 0.0f);
        case 2: return prb_activate(v, PRB_ACT_GELU_TANH);
        default: return v * ea_sigmoid(v);
    }
}

template <typename O, bool VEC>
__global__ void act_columns_kernel(O* __restrict__ out, long out_ld, const float* __restrict__ in, long in_ld,
                                   int n, int n_rows, int act) {
    prb_grid_launch_dependents();
    prb_grid_wait();
    const size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if constexpr (VEC) {
        const int n4 = n / 4;
        if (idx >= (size_t)n_rows * n4) return;
        const int t = (int)(idx / n4), i = (int)(idx - (size_t)t * n4) * 4;
        const float4 u = *reinterpret_cast<const float4*>(in + (size_t)t * in_ld + i);
        prb_store4(out + (size_t)t * out_ld + i, column_act(u.x, act), column_act(u.y, act), column_act(u.z, act),
                   column_act(u.w, act));
    } else {
        if (idx >= (size_t)n_rows * n) return;
        const int t = (int)(idx / n), i = (int)(idx - (size_t)t * n);
        out[(size_t)t * out_ld + i] = prb_from_float<O>(column_act(in[(size_t)t * in_ld + i], act));
    }
}
}  // namespace

PRB_API int prb_expert_act(void* out, long out_ld, const float* in, long in_ld, int gate_col, int up_col,
                           int router_col, int shared_gate_col, int shared_up_col, int shared_weight_col,
                           int n_rows, int experts, int identity, int top, int group, int shared, int renorm,
                           int act, float factor, const float* correction, float* x, long x_ld, int width,
                           const void* h, long h_ld, const float* norm_w, float eps, int dtype,
                           cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    const int all = experts + identity;
    if (experts < 0 || identity < 0 || all <= 0 || all > 2048 || top <= 0 || top > all || group <= 0 ||
        shared < 0 || act < 0 || act > 1)
        return PRB_E_SIZE;
    if (identity > 0 && (x == nullptr || width <= 0)) return PRB_E_ARG;
    const ExpertArgs a{out, out_ld, in, in_ld, gate_col, up_col, router_col, shared_gate_col, shared_up_col,
                       shared_weight_col, n_rows, experts, identity, top, group, shared, renorm, act, factor,
                       correction, x, x_ld, width, h, h_ld, norm_w, eps};
    const int columns = experts * group + shared;
    cudaError_t e;
    if (n_rows <= 64) {
        // a row a CTA and slice, four columns a thread where that leaves no more than 64 slices
        const int slices = columns < 1024 ? 1 : (columns + 1023) / 1024 > 64 ? 64 : (columns + 1023) / 1024;
        const dim3 grid(n_rows, slices);
        const size_t smem = (size_t)3 * all * sizeof(float);
        if (dtype == PRB_F32) e = prb_launch_dependent(expert_act_row_kernel<float>, grid, dim3(256), smem, stream, a);
        else if (dtype == PRB_BF16)
            e = prb_launch_dependent(expert_act_row_kernel<__nv_bfloat16>, grid, dim3(256), smem, stream, a);
        else return PRB_E_DTYPE;
    } else {
        const int groups = (n_rows + EA_ROWS - 1) / EA_ROWS;
        int slices = (columns + 1023) / 1024;
        if (slices < 1) slices = 1;
        while (slices > 1 && (long)groups * slices > 6L * prb_sm_count()) slices = (slices + 1) / 2;
        const dim3 grid(groups, slices);
        const size_t smem = (size_t)3 * EA_ROWS * all * sizeof(float);
        if (smem > 40 * 1024) {
            cudaFuncSetAttribute(expert_act_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
            cudaFuncSetAttribute(expert_act_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        }
        if (dtype == PRB_F32)
            e = prb_launch_maybe_early(false, expert_act_kernel<float>, grid, dim3(256), smem, stream, a);
        else if (dtype == PRB_BF16)
            e = prb_launch_maybe_early(false, expert_act_kernel<__nv_bfloat16>, grid, dim3(256), smem, stream, a);
        else return PRB_E_DTYPE;
    }
    return e == cudaSuccess ? 0 : (int)e;
}

// act 0: relu(.)^2, 1: relu, 2: gelu (tanh form), 3: silu; `in` points at the first column.
PRB_API int prb_act_columns(void* out, long out_ld, const float* in, long in_ld, int n, int n_rows, int act,
                            int out_dtype, cudaStream_t stream) {
    if (n <= 0 || n_rows <= 0) return 0;
    if (act < 0 || act > 3) return PRB_E_ARG;
    if (out_dtype != PRB_F32 && out_dtype != PRB_BF16) return PRB_E_DTYPE;
    const size_t esz = out_dtype == PRB_F32 ? 4 : 2, total = (size_t)n * n_rows;
    const bool vec = (n | in_ld | out_ld) % 4 == 0 && ((uintptr_t)in) % 16 == 0 && ((uintptr_t)out) % (4 * esz) == 0;
    const unsigned blocks = (unsigned)(((vec ? total / 4 : total) + 255) / 256);
    cudaError_t e;
#define ACTC(OT, V)                                                                                          \
    e = prb_launch_maybe_early(n_rows <= 64, act_columns_kernel<OT, V>, dim3(blocks), dim3(256), 0, stream,   \
                               (OT*)out, out_ld, in, in_ld, n, n_rows, act)
    if (out_dtype == PRB_F32) { if (vec) { ACTC(float, true); } else { ACTC(float, false); } }
    else { if (vec) { ACTC(__nv_bfloat16, true); } else { ACTC(__nv_bfloat16, false); } }
#undef ACTC
    return e == cudaSuccess ? 0 : (int)e;
}
