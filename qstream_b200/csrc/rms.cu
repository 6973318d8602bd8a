// RMS norms and the small kernels around a residual stream that is kept in 32-bit:
//
//   rmsnorm            y = x / sqrt(mean(x^2) + eps) * (offset + w)
//   residual_rmsnorm   x <- x + mult * y (32-bit, in place), and optionally h = rmsnorm(x) in the same pass
//   branch_norm        x <- x + norm_b(y) * w_b (in place), and optionally h = norm(x) * w in the same pass, with
//                      norm = layer norm without bias or RMS norm: layers that norm a branch before they add it
//   stream_tanh_norm   x <- x + sum of up to three branches (32-bit, in place), each with a factor and, if it has a
//                      weight, divided by its root mean square first; then up to two reads of the new x in the same
//                      pass: tanh(alpha x) * w + b (no statistics), or x itself
//   stream_norm        x <- x + sum of up to three branches (32-bit, in place), each with a factor (a branch whose rows
//                      are 0 apart is one vector for all tokens), and h = norm(x) * w + b of the new x in the same pass, with
//                      norm = layer norm or RMS norm
//   gated_group_norm   out = o / sqrt(mean_group(o^2) + eps) * w * act(gate), groups of consecutive elements
//                      (one group = the whole row, or one per head; group 0 = no norm, only the gate)
//   gated_act          out = act(a) * b for the two halves [a | b] of a fused projection (gated feed-forward)
//   activate           x <- act(x) in place
//   embedding_hashed   x = table[token] * scale + pair_table[hash(previous token, token)]
//   keep_last_rows     state[slot] = the last row each sequence brought in this step
//
// Every sum is taken in 32-bit in a fixed order (block_sum / warp_sum), whatever the storage types.
#include "common.cuh"

namespace {

// ----------------------------------------------------------------------------- rmsnorm

// One block per row, the row in shared memory as 32-bit floats.  With `y` the row is first updated:
// x <- x + mult * y, written back to `x_out` (which may be x itself).  `h_out` may be null (update only).
template <typename TX, typename TY, typename TH>
__global__ void residual_rmsnorm_kernel(TH* __restrict__ h_out, size_t ldh, TX* x_out, const TX* x, size_t ldx,
                                        const TY* __restrict__ y, size_t ldy, float mult,
                                        const void* __restrict__ w, int w_dtype, float offset, int D, float eps) {
    extern __shared__ float row[];
    __shared__ float scratch[33];
    grid_dep_launch();
    grid_dep_wait();
    const TX* src = x + (size_t)blockIdx.x * ldx;
    float s = 0.f;
    for (int i = threadIdx.x; i < D; i += blockDim.x) {
        float v = to_f32(src[i]);
        if (y) {
            v = fmaf(mult, to_f32(y[(size_t)blockIdx.x * ldy + i]), v);
            x_out[(size_t)blockIdx.x * ldx + i] = from_f32<TX>(v);
        }
        row[i] = v;
        s = fmaf(v, v, s);
    }
    if (!h_out) return;
    const float rstd = 1.0f / sqrtf(block_sum(s, scratch) / (float)D + eps);
    TH* dst = h_out + (size_t)blockIdx.x * ldh;
    for (int i = threadIdx.x; i < D; i += blockDim.x)
        dst[i] = from_f32<TH>(row[i] * rstd * (offset + load_as_f32(w, w_dtype, i)));
}

template <typename TX, typename TY, typename TH>
int launch_norm(void* h_out, long long ldh, void* x_out, const void* x, long long ldx, const void* y, long long ldy,
                float mult, const void* w, int w_dtype, float offset, int rows, int D, float eps, cudaStream_t stream) {
    const size_t smem = (size_t)D * sizeof(float);
    const int threads = D >= 4096 ? 512 : (D >= 1024 ? 256 : 128);
    auto kernel = residual_rmsnorm_kernel<TX, TY, TH>;
    if (smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return qs_fail(QS_ERR_INTERNAL, "rmsnorm: %s", cudaGetErrorString(e));
    }
    cudaError_t e = qs_launch_dependent(kernel, dim3(rows), dim3(threads), smem, stream, (TH*)h_out, (size_t)ldh,
                                        (TX*)x_out, (const TX*)x, (size_t)ldx, (const TY*)y, (size_t)ldy, mult, w, w_dtype,
                                        offset, D, eps);
    if (e != cudaSuccess) return qs_fail(QS_ERR_INTERNAL, "rmsnorm: %s", cudaGetErrorString(e));
    return qs_check_launch("rmsnorm");
}

// ----------------------------------------------------------------------------- norms around a branch

// One block per row, the row in shared memory as 32-bit floats.  The statistic of `v` over the row: with `center`
// mean and variance of the deviations (layer norm), without it the mean square (RMS norm); returns (mean, rstd).
__device__ __forceinline__ float2 row_statistic(const float* row, int D, float eps, int center, float* scratch) {
    float mean = 0.f;
    if (center) {
        float s = 0.f;
        for (int i = threadIdx.x; i < D; i += blockDim.x) s += row[i];
        mean = block_sum(s, scratch) / (float)D;
    }
    float q = 0.f;
    for (int i = threadIdx.x; i < D; i += blockDim.x) { const float d = row[i] - mean; q = fmaf(d, d, q); }
    const float var = block_sum(q, scratch) / (float)D;
    return make_float2(mean, 1.0f / sqrtf(var + eps));
}

// With y: x <- x + norm(y) * wy (wy null: x + y), written back in x's type.  With h_out: h = norm(x) * w, or, without
// w, x itself in h's type (a sublayer that reads the stream as it is).
// h_out may be x itself (a norm in place).  A thread reads back only what it wrote to `row`.
template <typename TX, typename TY, typename TH>
__global__ void branch_norm_kernel(TH* h_out, size_t ldh, TX* x, size_t ldx, const TY* __restrict__ y, size_t ldy,
                                   const void* __restrict__ wy, int wy_dtype, const void* __restrict__ w, int w_dtype,
                                   int D, float eps, int center) {
    extern __shared__ float row[];
    __shared__ float scratch[33];
    grid_dep_launch();
    grid_dep_wait();
    TX* xr = x + (size_t)blockIdx.x * ldx;
    if (y) {
        for (int i = threadIdx.x; i < D; i += blockDim.x) row[i] = to_f32(y[(size_t)blockIdx.x * ldy + i]);
        float2 st = make_float2(0.f, 1.f);
        if (wy) st = row_statistic(row, D, eps, center, scratch);
        for (int i = threadIdx.x; i < D; i += blockDim.x) {
            const float b = wy ? (row[i] - st.x) * st.y * load_as_f32(wy, wy_dtype, i) : row[i];
            const float v = to_f32(xr[i]) + b;
            xr[i] = from_f32<TX>(v);
            row[i] = v;
        }
    } else {
        for (int i = threadIdx.x; i < D; i += blockDim.x) row[i] = to_f32(xr[i]);
    }
    if (!h_out) return;
    TH* dst = h_out + (size_t)blockIdx.x * ldh;
    if (!w) {
        for (int i = threadIdx.x; i < D; i += blockDim.x) dst[i] = from_f32<TH>(row[i]);
        return;
    }
    const float2 st = row_statistic(row, D, eps, center, scratch);
    for (int i = threadIdx.x; i < D; i += blockDim.x)
        dst[i] = from_f32<TH>((row[i] - st.x) * st.y * load_as_f32(w, w_dtype, i));
}

template <typename TX, typename TY, typename TH>
int launch_branch_norm(void* h_out, long long ldh, void* x, long long ldx, const void* y, long long ldy, const void* wy,
                       int wy_dtype, const void* w, int w_dtype, int rows, int D, float eps, int center, cudaStream_t stream) {
    const size_t smem = (size_t)D * sizeof(float);
    const int threads = D >= 4096 ? 512 : (D >= 1024 ? 256 : 128);
    auto kernel = branch_norm_kernel<TX, TY, TH>;
    if (smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return qs_fail(QS_ERR_INTERNAL, "branch_norm: %s", cudaGetErrorString(e));
    }
    cudaError_t e = qs_launch_dependent(kernel, dim3(rows), dim3(threads), smem, stream, (TH*)h_out, (size_t)ldh, (TX*)x,
                                        (size_t)ldx, (const TY*)y, (size_t)ldy, wy, wy_dtype, w, w_dtype, D, eps, center);
    if (e != cudaSuccess) return qs_fail(QS_ERR_INTERNAL, "branch_norm: %s", cudaGetErrorString(e));
    return qs_check_launch("branch_norm");
}

// ----------------------------------------------------------------------------- branches into the stream, tanh norms

// Four neighbouring elements of a vector or a row, as stored.
template <typename T> struct FourOf;
template <> struct FourOf<float> { typedef float4 type; };
template <> struct FourOf<__nv_bfloat16> { typedef uint2 type; };
__device__ __forceinline__ float4 four_as_f32(float4 v) { return v; }
__device__ __forceinline__ float4 four_as_f32(uint2 v) {
    return make_float4(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xffff0000u), __uint_as_float(v.y << 16), __uint_as_float(v.y & 0xffff0000u));
}
__device__ __forceinline__ void store_four(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store_four(__nv_bfloat16* p, float4 v) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
}

struct StreamBranch { const float* y; size_t ld; const void* w; int w_dtype; float mult; };
struct TanhRead { void* h; size_t ld; const void* w; const void* b; int w_dtype, b_dtype; float alpha; };

// One block per row; V neighbouring columns per thread and round (V = 4: 16-byte aligned rows of whole fours).  The
// sums of squares of the normed branches are taken together.  A read without a weight hands on x itself.
template <typename TH, int V>
__global__ void stream_tanh_norm_kernel(float* __restrict__ x, size_t ldx, StreamBranch b0, StreamBranch b1, StreamBranch b2, TanhRead r0,
                                        TanhRead r1, int D, float eps) {
    __shared__ float part[3][32];
    grid_dep_launch();
    grid_dep_wait();
    const size_t t = blockIdx.x;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    const StreamBranch br[3] = {b0, b1, b2};
    float scale[3] = {b0.mult, b1.mult, b2.mult};
    if (b0.w || b1.w || b2.w) {
        float q[3] = {0.f, 0.f, 0.f};
        for (int i = threadIdx.x * V; i < D; i += blockDim.x * V)
#pragma unroll
            for (int k = 0; k < 3; ++k)
                if (br[k].w)
#pragma unroll
                    for (int v = 0; v < V; ++v) { const float y = br[k].y[t * br[k].ld + i + v]; q[k] = fmaf(y, y, q[k]); }
#pragma unroll
        for (int k = 0; k < 3; ++k) {
            q[k] = warp_sum(q[k]);
            if (lane == 0) part[k][warp] = q[k];
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < 3; ++k)
            if (br[k].w) {
                float total = 0.f;
                for (int i = 0; i < warps; ++i) total += part[k][i];
                scale[k] *= 1.0f / sqrtf(total / (float)D + eps);
            }
    }
    float* xr = x + t * ldx;
    for (int i = threadIdx.x * V; i < D; i += blockDim.x * V) {
        float xv[V];
#pragma unroll
        for (int v = 0; v < V; ++v) xv[v] = xr[i + v];
        if (b0.y) {
            float add[V];
#pragma unroll
            for (int v = 0; v < V; ++v) add[v] = 0.f;
#pragma unroll
            for (int k = 0; k < 3; ++k)
                if (br[k].y)
#pragma unroll
                    for (int v = 0; v < V; ++v) {
                        const float y = br[k].y[t * br[k].ld + i + v] * scale[k];
                        add[v] += br[k].w ? y * load_as_f32(br[k].w, br[k].w_dtype, i + v) : y;
                    }
#pragma unroll
            for (int v = 0; v < V; ++v) { xv[v] += add[v]; xr[i + v] = xv[v]; }
        }
        const TanhRead rd[2] = {r0, r1};
#pragma unroll
        for (int k = 0; k < 2; ++k)
            if (rd[k].h) {
                float h[V];
#pragma unroll
                for (int v = 0; v < V; ++v)
                    h[v] = rd[k].w ? fmaf(tanhf(rd[k].alpha * xv[v]), load_as_f32(rd[k].w, rd[k].w_dtype, i + v), load_as_f32(rd[k].b, rd[k].b_dtype, i + v))
                                   : xv[v];
                TH* dst = reinterpret_cast<TH*>(rd[k].h) + t * rd[k].ld + i;
                if (V == 4 && sizeof(TH) == 2) {
                    const __nv_bfloat162 lo = __floats2bfloat162_rn(h[0], h[1 % V]), hi = __floats2bfloat162_rn(h[2 % V], h[3 % V]);
                    *reinterpret_cast<uint2*>(dst) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
                } else {
#pragma unroll
                    for (int v = 0; v < V; ++v) dst[v] = from_f32<TH>(h[v]);
                }
            }
    }
}

// ----------------------------------------------------------------------------- branches into the stream, one norm

// One block per row; a thread holds PER pieces of four neighbouring columns in registers from the first load to the norm
// (16-byte aligned rows of whole fours, D <= 4 * PER * threads).  `settled`: weight and bias were complete before the
// previous kernel of the stream began; they are then fetched while that kernel still runs.
template <typename TH, typename TW, int PER>
__global__ void stream_norm_vec_kernel(float* __restrict__ x, size_t ldx, StreamBranch b0, StreamBranch b1, StreamBranch b2, TH* __restrict__ h,
                                       size_t ldh, const TW* __restrict__ w, const TW* __restrict__ b, int D, float eps, int center, int settled) {
    __shared__ float scratch[33];
    grid_dep_launch();
    if (!settled) grid_dep_wait();
    typedef typename FourOf<TW>::type W4;
    W4 wv[PER], bv[PER];
#pragma unroll
    for (int p = 0; p < PER; ++p) {
        const int c = (p * blockDim.x + threadIdx.x) * 4;
        if (c < D) {
            wv[p] = *reinterpret_cast<const W4*>(w + c);
            if (b) bv[p] = *reinterpret_cast<const W4*>(b + c);
        }
    }
    if (settled) grid_dep_wait();
    const size_t t = blockIdx.x;
    float* xr = x + t * ldx;
    float4 v[PER];
    float s = 0.f;
#pragma unroll
    for (int p = 0; p < PER; ++p) {
        const int c = (p * blockDim.x + threadIdx.x) * 4;
        v[p] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c < D) v[p] = *reinterpret_cast<const float4*>(xr + c);
    }
    if (b0.y) {
        const StreamBranch br[3] = {b0, b1, b2};
#pragma unroll
        for (int k = 0; k < 3; ++k) {
            if (!br[k].y) continue;
            const float* yr = br[k].y + t * br[k].ld;
            float4 y[PER];
#pragma unroll
            for (int p = 0; p < PER; ++p) {
                const int c = (p * blockDim.x + threadIdx.x) * 4;
                y[p] = make_float4(0.f, 0.f, 0.f, 0.f);
                if (c < D) y[p] = *reinterpret_cast<const float4*>(yr + c);
            }
#pragma unroll
            for (int p = 0; p < PER; ++p) {
                v[p].x = fmaf(br[k].mult, y[p].x, v[p].x); v[p].y = fmaf(br[k].mult, y[p].y, v[p].y);
                v[p].z = fmaf(br[k].mult, y[p].z, v[p].z); v[p].w = fmaf(br[k].mult, y[p].w, v[p].w);
            }
        }
#pragma unroll
        for (int p = 0; p < PER; ++p) {
            const int c = (p * blockDim.x + threadIdx.x) * 4;
            if (c < D) *reinterpret_cast<float4*>(xr + c) = v[p];
        }
    }
    float mean = 0.f;
    if (center) {
#pragma unroll
        for (int p = 0; p < PER; ++p) s += (v[p].x + v[p].y) + (v[p].z + v[p].w);
        mean = block_sum(s, scratch) / (float)D;
    }
    float q = 0.f;
#pragma unroll
    for (int p = 0; p < PER; ++p)
        if ((p * blockDim.x + threadIdx.x) * 4 < D) {
            v[p].x -= mean; v[p].y -= mean; v[p].z -= mean; v[p].w -= mean;
            q = fmaf(v[p].x, v[p].x, q); q = fmaf(v[p].y, v[p].y, q); q = fmaf(v[p].z, v[p].z, q); q = fmaf(v[p].w, v[p].w, q);
        }
    const float rstd = 1.0f / sqrtf(block_sum(q, scratch) / (float)D + eps);
#pragma unroll
    for (int p = 0; p < PER; ++p) {
        const int c = (p * blockDim.x + threadIdx.x) * 4;
        if (c >= D) continue;
        const float4 wf = four_as_f32(wv[p]), bf = b ? four_as_f32(bv[p]) : make_float4(0.f, 0.f, 0.f, 0.f);
        store_four(h + t * ldh + c, make_float4(fmaf(v[p].x * rstd, wf.x, bf.x), fmaf(v[p].y * rstd, wf.y, bf.y),
                                                fmaf(v[p].z * rstd, wf.z, bf.z), fmaf(v[p].w * rstd, wf.w, bf.w)));
    }
}

// The same for any width and alignment: the row in shared memory as 32-bit floats.
template <typename TH>
__global__ void stream_norm_kernel(float* __restrict__ x, size_t ldx, StreamBranch b0, StreamBranch b1, StreamBranch b2, TH* __restrict__ h, size_t ldh,
                                   const void* __restrict__ w, int w_dtype, const void* __restrict__ b, int b_dtype, int D, float eps, int center) {
    extern __shared__ float row[];
    __shared__ float scratch[33];
    grid_dep_launch();
    grid_dep_wait();
    const size_t t = blockIdx.x;
    const StreamBranch br[3] = {b0, b1, b2};
    for (int i = threadIdx.x; i < D; i += blockDim.x) {
        float v = x[t * ldx + i];
        if (b0.y) {
#pragma unroll
            for (int k = 0; k < 3; ++k)
                if (br[k].y) v = fmaf(br[k].mult, br[k].y[t * br[k].ld + i], v);
            x[t * ldx + i] = v;
        }
        row[i] = v;
    }
    const float2 st = row_statistic(row, D, eps, center, scratch);
    for (int i = threadIdx.x; i < D; i += blockDim.x)
        h[t * ldh + i] = from_f32<TH>(fmaf((row[i] - st.x) * st.y, load_as_f32(w, w_dtype, i), b ? load_as_f32(b, b_dtype, i) : 0.f));
}

// ----------------------------------------------------------------------------- gated group norm

// One block per row.  group == n: one norm over the row (block sum).  0 < group < n: a warp per group, groups dealt
// to the warps in turn.  group == 0: no norm.  Then * w[c] (if given) * act(gate[c / gate_span]) (if given; a span
// above 1 is one gate value for that many neighbouring elements, a head's say).
template <typename TI, typename TG, typename TO>
__global__ void gated_group_norm_kernel(TO* __restrict__ out, size_t ldo, const TI* __restrict__ o, size_t ldi,
                                        const void* __restrict__ w, int w_dtype, const TG* __restrict__ gate, size_t ldg,
                                        int gate_act, int n, int group, float eps, int gate_span) {
    extern __shared__ float rstd_of[];               // one per group (at least one)
    __shared__ float scratch[33];
    grid_dep_launch();
    grid_dep_wait();
    const TI* src = o + (size_t)blockIdx.x * ldi;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    if (group == n) {
        float s = 0.f;
        for (int i = threadIdx.x; i < n; i += blockDim.x) { const float v = to_f32(src[i]); s = fmaf(v, v, s); }
        const float total = block_sum(s, scratch);
        if (threadIdx.x == 0) rstd_of[0] = 1.0f / sqrtf(total / (float)n + eps);
    } else if (group > 0) {
        for (int g = warp; g * group < n; g += warps) {
            float s = 0.f;
            for (int i = lane; i < group; i += 32) { const float v = to_f32(src[g * group + i]); s = fmaf(v, v, s); }
            s = warp_sum(s);
            if (lane == 0) rstd_of[g] = 1.0f / sqrtf(s / (float)group + eps);
        }
    }
    __syncthreads();
    TO* dst = out + (size_t)blockIdx.x * ldo;
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
        float v = to_f32(src[i]);
        if (group > 0) v *= rstd_of[i / group];
        if (w) v *= load_as_f32(w, w_dtype, i);
        if (gate) v *= apply_activation(to_f32(gate[(size_t)blockIdx.x * ldg + (gate_span > 1 ? i / gate_span : i)]), gate_act);
        dst[i] = from_f32<TO>(v);
    }
}

template <typename TI, typename TG, typename TO>
int launch_gated(void* out, long long ldo, const void* o, long long ldi, const void* w, int w_dtype, const void* gate,
                 long long ldg, int gate_act, int rows, int n, int group, float eps, int gate_span, cudaStream_t stream) {
    const int n_groups = group > 0 ? n / group : 1;
    const int threads = n >= 2048 ? 256 : 128;
    cudaError_t e = qs_launch_dependent(gated_group_norm_kernel<TI, TG, TO>, dim3(rows), dim3(threads),
                                        (size_t)n_groups * sizeof(float), stream, (TO*)out, (size_t)ldo, (const TI*)o,
                                        (size_t)ldi, w, w_dtype, (const TG*)gate, (size_t)ldg, gate_act, n, group, eps, gate_span);
    if (e != cudaSuccess) return qs_fail(QS_ERR_INTERNAL, "gated_group_norm: %s", cudaGetErrorString(e));
    return qs_check_launch("gated_group_norm");
}

// ----------------------------------------------------------------------------- gated activation

// One row per blockIdx.x, a block of columns per blockIdx.y.  VEC (bfloat16, F a multiple of 8, 16-byte aligned
// rows): eight columns per thread as one 16-byte piece of each half.
template <typename T, bool VEC>
__global__ void gated_act_kernel(T* __restrict__ out, size_t ldo, const T* __restrict__ ab, size_t ldi, int F, int act) {
    grid_dep_launch();
    grid_dep_wait();
    const size_t r = blockIdx.x;
    const int c = (blockIdx.y * blockDim.x + threadIdx.x) * (VEC ? 8 : 1);
    if (c >= F) return;
    if (VEC) {
        const uint4 a = *reinterpret_cast<const uint4*>(ab + r * ldi + c), b = *reinterpret_cast<const uint4*>(ab + r * ldi + F + c);
        const uint32_t au[4] = {a.x, a.y, a.z, a.w}, bu[4] = {b.x, b.y, b.z, b.w};
        uint32_t o[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const float a0 = __uint_as_float(au[j] << 16), a1 = __uint_as_float(au[j] & 0xffff0000u);
            const float b0 = __uint_as_float(bu[j] << 16), b1 = __uint_as_float(bu[j] & 0xffff0000u);
            const __nv_bfloat162 p = __floats2bfloat162_rn(apply_activation(a0, act) * b0, apply_activation(a1, act) * b1);
            o[j] = *reinterpret_cast<const uint32_t*>(&p);
        }
        *reinterpret_cast<uint4*>(out + r * ldo + c) = make_uint4(o[0], o[1], o[2], o[3]);
    } else {
        const float a = to_f32(ab[r * ldi + c]), b = to_f32(ab[r * ldi + F + c]);
        out[r * ldo + c] = from_f32<T>(apply_activation(a, act) * b);
    }
}

// The clamped gated unit of two halves [a | b]: g = min(a, limit), u = clamp(b, -limit, limit),
// out = g * sigmoid(alpha * g) * (u + shift); 32-bit arithmetic, rounded once.  limit <= 0: no clamp.
__device__ __forceinline__ float clamped_glu(float g, float u, float limit, float alpha, float shift) {
    if (limit > 0.f) { g = fminf(g, limit); u = fminf(fmaxf(u, -limit), limit); }
    return g * sigmoid_f32(alpha * g) * (u + shift);
}

// VEC (bfloat16, F a multiple of 8, 16-byte aligned rows): eight columns per thread as one 16-byte piece of each half.
template <typename T, bool VEC>
__global__ void clamped_glu_kernel(T* __restrict__ out, size_t ldo, const T* __restrict__ ab, size_t ldi, int F, float limit,
                                   float alpha, float shift) {
    grid_dep_launch();
    grid_dep_wait();
    const size_t r = blockIdx.x;
    const int c = (blockIdx.y * blockDim.x + threadIdx.x) * (VEC ? 8 : 1);
    if (c >= F) return;
    if (VEC) {
        const uint4 a = *reinterpret_cast<const uint4*>(ab + r * ldi + c), b = *reinterpret_cast<const uint4*>(ab + r * ldi + F + c);
        const uint32_t au[4] = {a.x, a.y, a.z, a.w}, bu[4] = {b.x, b.y, b.z, b.w};
        uint32_t o[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const float a0 = __uint_as_float(au[j] << 16), a1 = __uint_as_float(au[j] & 0xffff0000u);
            const float b0 = __uint_as_float(bu[j] << 16), b1 = __uint_as_float(bu[j] & 0xffff0000u);
            const __nv_bfloat162 p = __floats2bfloat162_rn(clamped_glu(a0, b0, limit, alpha, shift), clamped_glu(a1, b1, limit, alpha, shift));
            o[j] = *reinterpret_cast<const uint32_t*>(&p);
        }
        *reinterpret_cast<uint4*>(out + r * ldo + c) = make_uint4(o[0], o[1], o[2], o[3]);
    } else {
        out[r * ldo + c] = from_f32<T>(clamped_glu(to_f32(ab[r * ldi + c]), to_f32(ab[r * ldi + F + c]), limit, alpha, shift));
    }
}

// x <- act(x), in 32-bit, rounded once: for activations that the matrix products' epilogues do not offer.
template <typename T>
__global__ void activate_kernel(T* __restrict__ x, size_t ld, int n, int act) {
    grid_dep_launch();
    grid_dep_wait();
    const int c = blockIdx.y * blockDim.x + threadIdx.x;
    if (c < n) x[(size_t)blockIdx.x * ld + c] = from_f32<T>(apply_activation_wide(to_f32(x[(size_t)blockIdx.x * ld + c]), act));
}

// ----------------------------------------------------------------------------- hashed-pair embedding

// x[t] = table[token] * scale + pair[row], row = (previous * mul_prev + token * mul_cur) mod buckets, and row
// `buckets` for a sequence's first token.  The previous token is the row above if it belongs to the same
// sequence, else what the sequence's earlier steps left in `last_token[slot]`.
template <typename TO, typename TT>
__global__ void embedding_hashed_kernel(TO* __restrict__ out, const TT* __restrict__ table, float scale,
                                        const TT* __restrict__ pair, long long buckets, long long mul_prev,
                                        long long mul_cur, const int32_t* __restrict__ tokens,
                                        const int32_t* __restrict__ tok_slot, const int32_t* __restrict__ tok_pos,
                                        const int32_t* __restrict__ last_token, size_t ld_last, int D, int V) {
    const int t = blockIdx.x;
    TO* dst = out + (size_t)t * D;
    const int slot = tok_slot[t];
    if (slot < 0) {
        for (int i = threadIdx.x; i < D; i += blockDim.x) dst[i] = from_f32<TO>(0.f);
        return;
    }
    int id = tokens[t];
    id = id < 0 ? 0 : (id >= V ? V - 1 : id);
    const TT* row = table + (size_t)id * D;
    const TT* prow = nullptr;
    if (pair) {
        long long r = buckets;
        if (tok_pos[t] > 0) {
            int prev = (t > 0 && tok_slot[t - 1] == slot) ? tokens[t - 1] : last_token[(size_t)slot * ld_last];
            prev = prev < 0 ? 0 : (prev >= V ? V - 1 : prev);
            r = ((long long)prev * mul_prev + (long long)id * mul_cur) % buckets;
            if (r < 0) r += buckets;
        }
        prow = pair + (size_t)r * D;
    }
    for (int i = threadIdx.x; i < D; i += blockDim.x) {
        float v = to_f32(row[i]) * scale;
        if (prow) v += to_f32(prow[i]);
        dst[i] = from_f32<TO>(v);
    }
}

// ----------------------------------------------------------------------------- keep last rows

// dst[slot] = the last row that each sequence of the step brought (rows of `row_bytes` bytes, 4-byte words).
__global__ void keep_last_rows_kernel(uint32_t* __restrict__ dst, size_t dst_words, const uint32_t* __restrict__ src,
                                      size_t src_words, int row_words, const int32_t* __restrict__ seq_start,
                                      const int32_t* __restrict__ seq_slot) {
    const int s = blockIdx.x;
    const int slot = seq_slot[s];
    const int a = seq_start[s], b = seq_start[s + 1];
    if (slot < 0 || b <= a) return;
    const uint32_t* from = src + (size_t)(b - 1) * src_words;
    uint32_t* to = dst + (size_t)slot * dst_words;
    for (int i = threadIdx.x; i < row_words; i += blockDim.x) to[i] = from[i];
}

}  // namespace

// h = rmsnorm(x) (y == null), or x_out = x + mult * y and h = rmsnorm(x_out) (h_out may then be null).
QS_API int qs_residual_rmsnorm(void* h_out, int h_dtype, long long ldh, void* x_out, const void* x, int x_dtype,
                               long long ldx, const void* y, int y_dtype, long long ldy, float mult, const void* w,
                               int w_dtype, float offset, int rows, int D, float eps, cudaStream_t stream) {
    if (rows == 0) return QS_OK;
    QS_REQUIRE(rows > 0 && D > 0, "rmsnorm: bad sizes rows=%d D=%d", rows, D);
    QS_REQUIRE(h_out || y, "rmsnorm: nothing to do");
    QS_REQUIRE(!h_out || w, "rmsnorm: a norm without a weight");
    QS_REQUIRE(!y || x_out, "rmsnorm: an update with nowhere to go");
    QS_REQUIRE((size_t)D * sizeof(float) <= 200 * 1024, "rmsnorm: width %d does not fit one block's shared memory", D);
    typedef __nv_bfloat16 bf16;
#define GO(TX, TY, TH) return launch_norm<TX, TY, TH>(h_out, ldh, x_out, x, ldx, y, ldy, mult, w, w_dtype, offset, rows, D, eps, stream)
    if (!y) y_dtype = x_dtype;
    if (!h_out) h_dtype = x_dtype;
    if (x_dtype == QS_F32 && y_dtype == QS_F32 && h_dtype == QS_F32) GO(float, float, float);
    if (x_dtype == QS_F32 && y_dtype == QS_F32 && h_dtype == QS_BF16) GO(float, float, bf16);
    if (x_dtype == QS_F32 && y_dtype == QS_BF16 && h_dtype == QS_BF16) GO(float, bf16, bf16);
    if (x_dtype == QS_F32 && y_dtype == QS_BF16 && h_dtype == QS_F32) GO(float, bf16, float);
    if (x_dtype == QS_BF16 && y_dtype == QS_BF16 && h_dtype == QS_BF16) GO(bf16, bf16, bf16);
#undef GO
    return qs_fail(QS_ERR_INVALID_INPUT, "rmsnorm: unsupported types x=%d y=%d h=%d", x_dtype, y_dtype, h_dtype);
}

// x <- x + norm(y) * wy (y given; wy null: plain sum) and h = norm(x) * w (h_out given; it may be x itself);
// `center` != 0: layer norm without bias, 0: RMS norm; statistics in 32-bit, eps inside the root.
QS_API int qs_branch_norm(void* h_out, int h_dtype, long long ldh, void* x, int x_dtype, long long ldx, const void* y,
                          int y_dtype, long long ldy, const void* wy, int wy_dtype, const void* w, int w_dtype, int rows,
                          int D, float eps, int center, cudaStream_t stream) {
    if (rows == 0) return QS_OK;
    QS_REQUIRE(rows > 0 && D > 0, "branch_norm: bad sizes rows=%d D=%d", rows, D);
    QS_REQUIRE(h_out || y, "branch_norm: nothing to do");
    QS_REQUIRE((size_t)D * sizeof(float) <= 200 * 1024, "branch_norm: width %d does not fit one block's shared memory", D);
    typedef __nv_bfloat16 bf16;
    if (!y) y_dtype = x_dtype;
    if (!h_out) h_dtype = x_dtype;
#define GO(TX, TY, TH) return launch_branch_norm<TX, TY, TH>(h_out, ldh, x, ldx, y, ldy, wy, wy_dtype, w, w_dtype, rows, D, eps, center, stream)
    if (x_dtype == QS_F32 && y_dtype == QS_F32 && h_dtype == QS_F32) GO(float, float, float);
    if (x_dtype == QS_F32 && y_dtype == QS_F32 && h_dtype == QS_BF16) GO(float, float, bf16);
    if (x_dtype == QS_F32 && y_dtype == QS_BF16 && h_dtype == QS_BF16) GO(float, bf16, bf16);
    if (x_dtype == QS_F32 && y_dtype == QS_BF16 && h_dtype == QS_F32) GO(float, bf16, float);
    if (x_dtype == QS_BF16 && y_dtype == QS_BF16 && h_dtype == QS_BF16) GO(bf16, bf16, bf16);
#undef GO
    return qs_fail(QS_ERR_INVALID_INPUT, "branch_norm: unsupported types x=%d y=%d h=%d", x_dtype, y_dtype, h_dtype);
}

// x [rows, D] float32 (row stride ldx).  Branches y0..y2 float32 or null (a null one ends the list), with factors m0..m2
// and, for a branch that is divided by its root mean square over D first, a weight w0..w2.  Reads h0, h1 (null: none) of
// type `h_dtype`: tanh(alpha x) * w + b, or, with a null weight, x.
QS_API int qs_stream_tanh_norm(float* x, long long ldx, int rows, int D, float eps, const float* y0, long long ld0, float m0, const void* w0,
                               int w0_dtype, const float* y1, long long ld1, float m1, const void* w1, int w1_dtype, const float* y2,
                               long long ld2, float m2, const void* w2, int w2_dtype, int h_dtype, void* h0, long long ldh0, float alpha0,
                               const void* nw0, int nw0_dtype, const void* nb0, int nb0_dtype, void* h1, long long ldh1, float alpha1,
                               const void* nw1, int nw1_dtype, const void* nb1, int nb1_dtype, cudaStream_t stream) {
    if (rows == 0) return QS_OK;
    QS_REQUIRE(rows > 0 && D > 0 && x, "stream_tanh_norm: bad sizes");
    QS_REQUIRE((y0 || !y1) && (y1 || !y2), "stream_tanh_norm: a branch behind a missing one");
    QS_REQUIRE((!w0 || y0) && (!w1 || y1) && (!w2 || y2), "stream_tanh_norm: a weight without its branch");
    QS_REQUIRE((!nw0 || (h0 && nb0)) && (!nw1 || (h1 && nb1)), "stream_tanh_norm: a norm lacks its output or its shift");
    QS_REQUIRE(h_dtype == QS_F32 || h_dtype == QS_BF16, "stream_tanh_norm: unknown dtype %d", h_dtype);
    const StreamBranch b0 = {y0, (size_t)ld0, w0, w0_dtype, m0}, b1 = {y1, (size_t)ld1, w1, w1_dtype, m1}, b2 = {y2, (size_t)ld2, w2, w2_dtype, m2};
    const TanhRead r0 = {h0, (size_t)ldh0, nw0, nb0, nw0_dtype, nb0_dtype, alpha0}, r1 = {h1, (size_t)ldh1, nw1, nb1, nw1_dtype, nb1_dtype, alpha1};
    auto fits = [](const void* p, long long ld) { return !p || (((uintptr_t)p % 16) == 0 && ld % 4 == 0); };
    const bool vec = D % 4 == 0 && fits(x, ldx) && fits(y0, ld0) && fits(y1, ld1) && fits(y2, ld2) && fits(h0, ldh0) && fits(h1, ldh1);
    const int items = vec ? (D + 3) / 4 : D;
    const int threads = items >= 512 ? 512 : (items >= 256 ? 256 : 128);
    cudaError_t e;
#define GO(TH, V) e = qs_launch_dependent(stream_tanh_norm_kernel<TH, V>, dim3(rows), dim3(threads), 0, stream, x, (size_t)ldx, b0, b1, b2, r0, r1, D, eps)
    if (h_dtype == QS_F32) { if (vec) GO(float, 4); else GO(float, 1); }
    else { if (vec) GO(__nv_bfloat16, 4); else GO(__nv_bfloat16, 1); }
#undef GO
    if (e != cudaSuccess) return qs_fail(QS_ERR_INTERNAL, "stream_tanh_norm: %s", cudaGetErrorString(e));
    return qs_check_launch("stream_tanh_norm");
}

// x [rows, D] float32 (row stride ldx).  Branches y0..y2 float32 or null (a null one ends the list), with factors m0..m2; a row
// stride of 0 gives every row the same vector.  h [rows, D] of type `h_dtype` = norm(x) * w + b (b may be null); `center` != 0:
// layer norm, 0: RMS norm; statistics in 32-bit, eps inside the root.
QS_API int qs_stream_norm(float* x, long long ldx, int rows, int D, float eps, int center, const float* y0, long long ld0, float m0,
                          const float* y1, long long ld1, float m1, const float* y2, long long ld2, float m2, int h_dtype, void* h,
                          long long ldh, const void* w, int w_dtype, const void* b, int b_dtype, int settled, cudaStream_t stream) {
    if (rows == 0) return QS_OK;
    QS_REQUIRE(rows > 0 && D > 0 && x && h && w, "stream_norm: bad sizes");
    QS_REQUIRE((y0 || !y1) && (y1 || !y2), "stream_norm: a branch behind a missing one");
    QS_REQUIRE(h_dtype == QS_F32 || h_dtype == QS_BF16, "stream_norm: unknown dtype %d", h_dtype);
    QS_REQUIRE((size_t)D * sizeof(float) <= 200 * 1024, "stream_norm: width %d does not fit one block's shared memory", D);
    typedef __nv_bfloat16 bf16;
    const StreamBranch b0 = {y0, (size_t)ld0, nullptr, 0, m0}, b1 = {y1, (size_t)ld1, nullptr, 0, m1}, b2 = {y2, (size_t)ld2, nullptr, 0, m2};
    auto fits = [](const void* p, long long ld) { return !p || (((uintptr_t)p % 16) == 0 && ld % 4 == 0); };
    const bool vec = D % 4 == 0 && D <= 16384 && fits(x, ldx) && fits(y0, ld0) && fits(y1, ld1) && fits(y2, ld2) && fits(h, ldh) && fits(w, 0) &&
                     fits(b, 0) && (!b || b_dtype == w_dtype);
    cudaError_t e = cudaSuccess;
    if (vec) {
        // many rows: few threads with several loads in flight each; few rows: as many threads as help
        const int per = rows >= 256 ? (D >= 2048 ? 4 : (D >= 1024 ? 2 : 1)) : (D <= 2048 ? 1 : (D <= 4096 ? 2 : 4));
        const int threads = ((D / 4 + per - 1) / per + 31) / 32 * 32;
#define GOV(TH, TW, PER) e = qs_launch_dependent(stream_norm_vec_kernel<TH, TW, PER>, dim3(rows), dim3(threads), 0, stream, x, (size_t)ldx, b0, b1, b2, \
        (TH*)h, (size_t)ldh, (const TW*)w, (const TW*)b, D, eps, center, settled)
#define GOP(TH, TW) do { if (per == 1) GOV(TH, TW, 1); else if (per == 2) GOV(TH, TW, 2); else GOV(TH, TW, 4); } while (0)
        if (h_dtype == QS_F32) { if (w_dtype == QS_F32) GOP(float, float); else GOP(float, bf16); }
        else { if (w_dtype == QS_F32) GOP(bf16, float); else GOP(bf16, bf16); }
#undef GOP
#undef GOV
    } else {
        const size_t smem = (size_t)D * sizeof(float);
        const int threads = D >= 4096 ? 512 : (D >= 1024 ? 256 : 128);
#define GO(TH) do { if (smem > 48 * 1024) e = cudaFuncSetAttribute(stream_norm_kernel<TH>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        if (e == cudaSuccess) e = qs_launch_dependent(stream_norm_kernel<TH>, dim3(rows), dim3(threads), smem, stream, x, (size_t)ldx, b0, b1, b2, \
            (TH*)h, (size_t)ldh, w, w_dtype, b, b_dtype, D, eps, center); } while (0)
        if (h_dtype == QS_F32) GO(float); else GO(bf16);
#undef GO
    }
    if (e != cudaSuccess) return qs_fail(QS_ERR_INTERNAL, "stream_norm: %s", cudaGetErrorString(e));
    return qs_check_launch("stream_norm");
}

QS_API int qs_gated_group_norm(void* out, int out_dtype, long long ldo, const void* o, int o_dtype, long long ldi,
                               const void* w, int w_dtype, const void* gate, int gate_dtype, long long ldg,
                               int gate_act, int rows, int n, int group, float eps, int gate_span, cudaStream_t stream) {
    if (rows == 0) return QS_OK;
    QS_REQUIRE(rows > 0 && n > 0 && group >= 0 && (group == 0 || n % group == 0),
               "gated_group_norm: bad sizes rows=%d n=%d group=%d", rows, n, group);
    QS_REQUIRE(gate_span >= 1 && n % gate_span == 0, "gated_group_norm: %d elements in spans of %d", n, gate_span);
    typedef __nv_bfloat16 bf16;
    if (!gate) gate_dtype = out_dtype;
#define GO(TI, TG, TO) return launch_gated<TI, TG, TO>(out, ldo, o, ldi, w, w_dtype, gate, ldg, gate_act, rows, n, group, eps, gate_span, stream)
    if (o_dtype == QS_F32 && gate_dtype == QS_F32 && out_dtype == QS_F32) GO(float, float, float);
    if (o_dtype == QS_F32 && gate_dtype == QS_BF16 && out_dtype == QS_BF16) GO(float, bf16, bf16);
    if (o_dtype == QS_F32 && gate_dtype == QS_F32 && out_dtype == QS_BF16) GO(float, float, bf16);
    if (o_dtype == QS_BF16 && gate_dtype == QS_BF16 && out_dtype == QS_BF16) GO(bf16, bf16, bf16);
#undef GO
    return qs_fail(QS_ERR_INVALID_INPUT, "gated_group_norm: unsupported types o=%d gate=%d out=%d", o_dtype, gate_dtype, out_dtype);
}

QS_API int qs_gated_act(void* out, long long ldo, const void* ab, long long ldi, int dtype, int rows, int F, int act,
                        cudaStream_t stream) {
    if (rows == 0) return QS_OK;
    QS_REQUIRE(rows > 0 && F > 0 && ldi >= 2 * (long long)F && ldo >= F, "gated_act: bad sizes rows=%d F=%d", rows, F);
    typedef __nv_bfloat16 bf16;
    cudaError_t e;
    if (dtype == QS_BF16 && F % 8 == 0 && ldi % 8 == 0 && ldo % 8 == 0 && ((uintptr_t)ab % 16) == 0 && ((uintptr_t)out % 16) == 0) {
        const int threads = F >= 2048 ? 256 : 64;
        const int by = (F / 8 + threads - 1) / threads;
        QS_REQUIRE(by <= 65535, "gated_act: %d columns exceed the grid", F);
        e = qs_launch_dependent(gated_act_kernel<bf16, true>, dim3(rows, by), dim3(threads), 0, stream, (bf16*)out, (size_t)ldo,
                                (const bf16*)ab, (size_t)ldi, F, act);
    } else {
        const int by = (F + 255) / 256;
        QS_REQUIRE(by <= 65535, "gated_act: %d columns exceed the grid", F);
        if (dtype == QS_F32)
            e = qs_launch_dependent(gated_act_kernel<float, false>, dim3(rows, by), dim3(256), 0, stream, (float*)out, (size_t)ldo,
                                    (const float*)ab, (size_t)ldi, F, act);
        else if (dtype == QS_BF16)
            e = qs_launch_dependent(gated_act_kernel<bf16, false>, dim3(rows, by), dim3(256), 0, stream, (bf16*)out, (size_t)ldo,
                                    (const bf16*)ab, (size_t)ldi, F, act);
        else return qs_fail(QS_ERR_INVALID_INPUT, "gated_act: unknown dtype %d", dtype);
    }
    if (e != cudaSuccess) return qs_fail(QS_ERR_INTERNAL, "gated_act: %s", cudaGetErrorString(e));
    return qs_check_launch("gated_act");
}

QS_API int qs_clamped_glu(void* out, long long ldo, const void* ab, long long ldi, int dtype, int rows, int F, float limit,
                          float alpha, float shift, cudaStream_t stream) {
    if (rows == 0) return QS_OK;
    QS_REQUIRE(rows > 0 && F > 0 && ldi >= 2 * (long long)F && ldo >= F, "clamped_glu: bad sizes rows=%d F=%d", rows, F);
    typedef __nv_bfloat16 bf16;
    cudaError_t e;
    if (dtype == QS_BF16 && F % 8 == 0 && ldi % 8 == 0 && ldo % 8 == 0 && ((uintptr_t)ab % 16) == 0 && ((uintptr_t)out % 16) == 0) {
        const int threads = F >= 2048 ? 256 : 64;
        const int by = (F / 8 + threads - 1) / threads;
        QS_REQUIRE(by <= 65535, "clamped_glu: %d columns exceed the grid", F);
        e = qs_launch_dependent(clamped_glu_kernel<bf16, true>, dim3(rows, by), dim3(threads), 0, stream, (bf16*)out, (size_t)ldo,
                                (const bf16*)ab, (size_t)ldi, F, limit, alpha, shift);
    } else {
        const int threads = F >= 256 ? 256 : 64;
        const int by = (F + threads - 1) / threads;
        QS_REQUIRE(by <= 65535, "clamped_glu: %d columns exceed the grid", F);
        if (dtype == QS_F32)
            e = qs_launch_dependent(clamped_glu_kernel<float, false>, dim3(rows, by), dim3(threads), 0, stream, (float*)out, (size_t)ldo,
                                    (const float*)ab, (size_t)ldi, F, limit, alpha, shift);
        else if (dtype == QS_BF16)
            e = qs_launch_dependent(clamped_glu_kernel<bf16, false>, dim3(rows, by), dim3(threads), 0, stream, (bf16*)out, (size_t)ldo,
                                    (const bf16*)ab, (size_t)ldi, F, limit, alpha, shift);
        else return qs_fail(QS_ERR_INVALID_INPUT, "clamped_glu: unknown dtype %d", dtype);
    }
    if (e != cudaSuccess) return qs_fail(QS_ERR_INTERNAL, "clamped_glu: %s", cudaGetErrorString(e));
    return qs_check_launch("clamped_glu");
}

QS_API int qs_activate(void* x, long long ld, int dtype, int rows, int n, int act, cudaStream_t stream) {
    if (rows == 0 || n == 0) return QS_OK;
    QS_REQUIRE(rows > 0 && n > 0 && ld >= n && (n + 255) / 256 <= 65535, "activate: bad sizes rows=%d n=%d", rows, n);
    cudaError_t e;
    if (dtype == QS_F32)
        e = qs_launch_dependent(activate_kernel<float>, dim3(rows, (n + 255) / 256), dim3(256), 0, stream, (float*)x, (size_t)ld, n, act);
    else if (dtype == QS_BF16)
        e = qs_launch_dependent(activate_kernel<__nv_bfloat16>, dim3(rows, (n + 255) / 256), dim3(256), 0, stream,
                                (__nv_bfloat16*)x, (size_t)ld, n, act);
    else return qs_fail(QS_ERR_INVALID_INPUT, "activate: unknown dtype %d", dtype);
    if (e != cudaSuccess) return qs_fail(QS_ERR_INTERNAL, "activate: %s", cudaGetErrorString(e));
    return qs_check_launch("activate");
}

QS_API int qs_embedding_hashed(void* out, int out_dtype, const void* table, const void* pair, int table_dtype, float scale,
                               long long buckets, long long mul_prev, long long mul_cur, const int32_t* tokens,
                               const int32_t* tok_slot, const int32_t* tok_pos, const int32_t* last_token, long long ld_last,
                               int T, int D, int V, cudaStream_t stream) {
    if (T == 0) return QS_OK;
    QS_REQUIRE(T > 0 && D > 0 && V > 0, "embedding: bad sizes T=%d D=%d V=%d", T, D, V);
    QS_REQUIRE(!pair || (buckets > 0 && last_token), "embedding: a pair table needs buckets and the sequences' last tokens");
    const int threads = D >= 1024 ? 256 : 128;
#define LAUNCH(TO, TT) embedding_hashed_kernel<TO, TT><<<T, threads, 0, stream>>>((TO*)out, (const TT*)table, scale, \
        (const TT*)pair, buckets, mul_prev, mul_cur, tokens, tok_slot, tok_pos, last_token, (size_t)ld_last, D, V)
    if (out_dtype == QS_F32 && table_dtype == QS_F32) LAUNCH(float, float);
    else if (out_dtype == QS_F32 && table_dtype == QS_BF16) LAUNCH(float, __nv_bfloat16);
    else if (out_dtype == QS_BF16 && table_dtype == QS_BF16) LAUNCH(__nv_bfloat16, __nv_bfloat16);
    else return qs_fail(QS_ERR_INVALID_INPUT, "embedding: unsupported types out=%d table=%d", out_dtype, table_dtype);
#undef LAUNCH
    return qs_check_launch("embedding_hashed");
}

QS_API int qs_keep_last_rows(void* dst, long long dst_bytes, const void* src, long long src_bytes, int row_bytes,
                             const int32_t* seq_start, const int32_t* seq_slot, int n_seq, cudaStream_t stream) {
    if (n_seq == 0) return QS_OK;
    QS_REQUIRE(n_seq > 0 && row_bytes > 0 && row_bytes % 4 == 0 && dst_bytes % 4 == 0 && src_bytes % 4 == 0 &&
               ((uintptr_t)dst % 4) == 0 && ((uintptr_t)src % 4) == 0, "keep_last_rows: rows must be whole 4-byte words");
    const int words = row_bytes / 4;
    keep_last_rows_kernel<<<n_seq, words >= 256 ? 256 : (words >= 64 ? 64 : 32), 0, stream>>>(
        (uint32_t*)dst, (size_t)dst_bytes / 4, (const uint32_t*)src, (size_t)src_bytes / 4, words, seq_start, seq_slot);
    return qs_check_launch("keep_last_rows");
}
