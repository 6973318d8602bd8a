// Recurrences whose state belongs to a channel, the short convolutions in front of them, and what surrounds Mamba-2's.
//
//   short convolution (causal, one filter per channel):
//       y_t[c] = act(bias[c] + sum_j taps[c][n - 1 - j] x_{t-j}[c])         x is zero before the sequence's start
//   selective scan (Mamba): N states per channel,
//       dt = softplus(raw),  S[c][n] <- exp(dt_c A[c][n]) S[c][n] + dt_c x_c B_n,  y_c = sum_n S[c][n] C_n + D_c x_c,
//       out = y silu(z)
//   gated linear recurrent unit (RG-LRU): one state per channel,
//       r, i = sigmoid(gate + bias),  log a = -8 r softplus(lam),  S <- a S + sqrt(1 - a^2) i u,  out = S gelu_tanh(y)
//   Mamba-2: the gates of its matrix recurrence (`ssd_gates`; the recurrence itself is state_scan's "ssd"), and
//       `ssd_output`: v = (o + D_h x) silu(z), divided by the root mean square of each of equal parts, times a weight
//
// States live in 32-bit per slot, start at zero, and are read at the start of a step and written back at its end; the
// convolution's last n - 1 inputs of a sequence are state too.  Everything that enters a recurrence besides the inputs
// x, u, B, C (the projections' and convolutions' own type) is 32-bit.
//
// Both scans walk a sequence's tokens in order.  A long prompt is cut into chunks that run side by side: PHASE 1 walks
// every chunk from an empty state and leaves the state it ends with and the sum of the logarithms of its decays; a
// prefix kernel walks each sequence's chunks and gives each the state it starts from (the slot the last one); PHASE 2
// walks every chunk from that state for the outputs.  PHASE 0: a sequence in order, from and to its slot.
#include "common.cuh"

namespace {

// ----------------------------------------------------------------------------- short convolution

constexpr int CONV_TOKENS = 8;          // tokens per block
constexpr int AHEAD = 8;                // loads in flight per thread where a chain is walked

template <typename T, int V> __device__ __forceinline__ void load_row(const T* __restrict__ p, float (&f)[V]) {
    if (V == 8) {
        float g[8];
        load8_as_f32(p, sizeof(T) == 4 ? QS_F32 : QS_BF16, 0, g);
#pragma unroll
        for (int v = 0; v < V; ++v) f[v] = g[v];
    } else {
#pragma unroll
        for (int v = 0; v < V; ++v) f[v] = to_f32(p[v]);
    }
}

template <typename T, int V> __device__ __forceinline__ void store_row(T* __restrict__ p, const float (&f)[V]) {
    if (V == 8 && sizeof(T) == 2) {
        uint32_t w[4];
#pragma unroll
        for (int v = 0; v < 4; ++v) {
            const __nv_bfloat162 b = __floats2bfloat162_rn(f[2 * v < V ? 2 * v : 0], f[2 * v + 1 < V ? 2 * v + 1 : 0]);
            w[v] = *reinterpret_cast<const uint32_t*>(&b);
        }
        *reinterpret_cast<uint4*>(p) = make_uint4(w[0], w[1], w[2], w[3]);
    } else {
#pragma unroll
        for (int v = 0; v < V; ++v) p[v] = from_f32<T>(f[v]);
    }
}

template <typename T, int V> struct alignas(sizeof(T) * V >= 16 ? 16 : sizeof(T)) RowPack { T v[V]; };

// The activation behind a convolution; a bfloat16 result takes silu on the fast exponential and division (off by about
// 1e-6 of the value).
template <typename T> __device__ __forceinline__ float conv_activation(float v, int act) {
    if (sizeof(T) == 2 && act == QS_ACT_SILU) return __fdividef(v, 1.0f + __expf(-v));
    return apply_activation(v, act);
}

// Prompts: blockIdx.x CONV_TOKENS rows of the packed batch, blockIdx.y a range of channels, V neighbouring channels per
// thread.  A token's predecessors lie in the rows above it if they came with this step, else in `held` [slot][n - 1][C].
// NT > 0: the number of taps, whose weights then stay in registers.
template <typename T, int V, int NT>
__global__ void short_conv_kernel(T* __restrict__ out, size_t ldo, const T* __restrict__ x, size_t ldx,
                                  const void* __restrict__ taps, int w_dtype, const void* __restrict__ bias, int b_dtype,
                                  int any_taps, const T* __restrict__ held, size_t slot_stride,
                                  const int32_t* __restrict__ tok_slot, const int32_t* __restrict__ tok_pos, int T_rows, int C,
                                  int act) {
    const int n_taps = NT > 0 ? NT : any_taps;
    __shared__ int s_slot[CONV_TOKENS], s_here[CONV_TOKENS];
    __shared__ int s_plain;
    if (threadIdx.x == 0) s_plain = 1;
    __syncthreads();
    grid_dep_launch();
    grid_dep_wait();
    const int t0 = blockIdx.x * CONV_TOKENS, nt = min(CONV_TOKENS, T_rows - t0);
    if (threadIdx.x < nt) {
        const int t = t0 + threadIdx.x, slot = tok_slot[t], pos = tok_pos[t];
        int here = 0;                                   // predecessors that came with this step, up to n - 1
        if (slot >= 0)
            while (here < n_taps - 1 && t - here - 1 >= 0 && tok_slot[t - here - 1] == slot && tok_pos[t - here - 1] == pos - here - 1) ++here;
        s_slot[threadIdx.x] = slot;
        s_here[threadIdx.x] = here;
        if (slot < 0 || here < n_taps - 1 || nt < CONV_TOKENS) s_plain = 0;
    }
    __syncthreads();
    const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
    if (c >= C) return;
    float b[V];
    float wreg[NT > 0 ? NT : 1][V];                     // [j]: the weight of the input j tokens back
    if (NT > 0 && V == 8) {                             // the V channels' taps (and biases) lie side by side: 16-byte loads
        float flat[(NT > 0 ? NT : 1) * 8], b8[8];
#pragma unroll
        for (int i = 0; i < (NT > 0 ? NT : 1); ++i) {
            float piece[8];
            load8_as_f32(taps, w_dtype, c * NT + 8 * i, piece);
#pragma unroll
            for (int v = 0; v < 8; ++v) flat[8 * i + v] = piece[v];
        }
        if (bias) load8_as_f32(bias, b_dtype, c, b8);
#pragma unroll
        for (int v = 0; v < V; ++v) {
            b[v] = bias ? b8[v % 8] : 0.f;
#pragma unroll
            for (int j = 0; j < (NT > 0 ? NT : 1); ++j) wreg[j][v] = flat[(v % 8) * (NT > 0 ? NT : 1) + (NT > 0 ? NT : 1) - 1 - j];
        }
    } else {
#pragma unroll
        for (int v = 0; v < V; ++v) b[v] = bias ? load_as_f32(bias, b_dtype, c + v) : 0.f;
    }
    if (NT > 1 && s_plain) {
        // a full tile of one sequence whose predecessors all came with this step: every row once, all loads in flight
        RowPack<T, V> rows[CONV_TOKENS + (NT > 1 ? NT - 1 : 0)];
#pragma unroll
        for (int i = 0; i < CONV_TOKENS + (NT > 1 ? NT - 1 : 0); ++i)
            rows[i] = *reinterpret_cast<const RowPack<T, V>*>(x + (size_t)(t0 - (NT > 1 ? NT - 1 : 0) + i) * ldx + c);
#pragma unroll
        for (int tt = 0; tt < CONV_TOKENS; ++tt) {
            float acc[V];
#pragma unroll
            for (int v = 0; v < V; ++v) acc[v] = b[v];
#pragma unroll
            for (int j = 0; j < (NT > 1 ? NT : 1); ++j)
#pragma unroll
                for (int v = 0; v < V; ++v) acc[v] = fmaf(wreg[j][v], to_f32(rows[tt + (NT > 1 ? NT - 1 : 0) - j].v[v]), acc[v]);
#pragma unroll
            for (int v = 0; v < V; ++v) acc[v] = conv_activation<T>(acc[v], act);
            store_row<T, V>(out + (size_t)(t0 + tt) * ldo + c, acc);
        }
        return;
    }
    for (int tt = 0; tt < nt; ++tt) {
        const int t = t0 + tt, slot = s_slot[tt], here = s_here[tt];
        float acc[V];
#pragma unroll
        for (int v = 0; v < V; ++v) acc[v] = slot >= 0 ? b[v] : 0.f;
        if (slot >= 0) {
#pragma unroll
            for (int j = 0; j < n_taps; ++j) {          // the input j tokens back meets tap number n - 1 - j
                const T* src = j <= here ? x + (size_t)(t - j) * ldx + c
                                         : held + (size_t)slot * slot_stride + (size_t)(n_taps - 1 - (j - here)) * C + c;
                float xv[V];
                load_row<T, V>(src, xv);
#pragma unroll
                for (int v = 0; v < V; ++v)
                    acc[v] = fmaf(NT > 0 ? wreg[NT > 0 ? j : 0][v] : load_as_f32(taps, w_dtype, (size_t)(c + v) * n_taps + n_taps - 1 - j), xv[v], acc[v]);
            }
#pragma unroll
            for (int v = 0; v < V; ++v) acc[v] = conv_activation<T>(acc[v], act);
        }
        store_row<T, V>(out + (size_t)t * ldo + c, acc);
    }
}

// After a prompt: the last n - 1 inputs of what each sequence's slot held and the step brought.  A thread reads a row of
// its channel before it overwrites it (rows in rising order).
template <typename T>
__global__ void conv_keep_kernel(T* __restrict__ held, size_t slot_stride, const T* __restrict__ x, size_t ldx, int C, int n_taps,
                                 const int32_t* __restrict__ seq_start, const int32_t* __restrict__ seq_slot) {
    grid_dep_launch();
    grid_dep_wait();
    const int s = blockIdx.x, slot = seq_slot[s];
    const int t0 = seq_start[s], n = seq_start[s + 1] - t0, keep = n_taps - 1;
    if (slot < 0 || n <= 0) return;
    T* mine = held + (size_t)slot * slot_stride;
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < C; c += gridDim.y * blockDim.x)
        for (int j = 0; j < keep; ++j) {
            const int idx = n - keep + j;
            mine[(size_t)j * C + c] = idx >= 0 ? x[(size_t)(t0 + idx) * ldx + c] : mine[(size_t)(j + n) * C + c];
        }
}

// Decode: row t is one token of the sequence in tok_slot[t]; the convolution and the new state in one pass, a thread
// per channel (it alone reads and writes its channel's state).
template <typename T>
__global__ void short_conv_step_kernel(T* __restrict__ out, size_t ldo, const T* __restrict__ x, size_t ldx,
                                       const void* __restrict__ taps, int w_dtype, const void* __restrict__ bias, int b_dtype,
                                       int n_taps, T* __restrict__ held, size_t slot_stride, const int32_t* __restrict__ tok_slot,
                                       int C, int act) {
    grid_dep_launch();
    grid_dep_wait();
    const int t = blockIdx.x, slot = tok_slot[t];
    const int c = blockIdx.y * blockDim.x + threadIdx.x;
    if (c >= C) return;
    if (slot < 0) { out[(size_t)t * ldo + c] = from_f32<T>(0.f); return; }
    const T now = x[(size_t)t * ldx + c];
    T* mine = held + (size_t)slot * slot_stride + c;
    float acc = fmaf(load_as_f32(taps, w_dtype, (size_t)c * n_taps + n_taps - 1), to_f32(now), bias ? load_as_f32(bias, b_dtype, c) : 0.f);
    for (int j = 1; j < n_taps; ++j)                    // row n - 1 - j of the state is the input j tokens back
        acc = fmaf(load_as_f32(taps, w_dtype, (size_t)c * n_taps + n_taps - 1 - j), to_f32(mine[(size_t)(n_taps - 1 - j) * C]), acc);
    for (int j = 0; j + 1 < n_taps - 1; ++j) mine[(size_t)j * C] = mine[(size_t)(j + 1) * C];
    if (n_taps > 1) mine[(size_t)(n_taps - 2) * C] = now;
    out[(size_t)t * ldo + c] = from_f32<T>(apply_activation(acc, act));
}

// ----------------------------------------------------------------------------- selective scan

constexpr int SCAN_TILE = 16;           // tokens staged in shared memory at a time
constexpr int SCAN_THREADS = 256;
// A decay a = 2^(dt a2) acts as S <- S + (a - 1) S: for decays close to one the error of a - 1 is small against it, where
// the error of a itself would add up over the tokens a state remembers.  The 32-bit engine takes a - 1 with expm1; the
// bfloat16 engine, whose inputs carry far larger errors, from the power of two.
template <typename T> __device__ __forceinline__ float decay_minus_one(float dt, float a2);
template <> __device__ __forceinline__ float decay_minus_one<float>(float dt, float a) { return expm1f(dt * a); }
template <> __device__ __forceinline__ float decay_minus_one<__nv_bfloat16>(float dt, float a2) { return exp2f(dt * a2) - 1.0f; }

// A block owns SCAN_THREADS >> ln_log2 channels of one sequence (or chunk); the 1 << ln_log2 lanes of a channel are
// neighbours in a warp and own SN states each, in groups of four dealt to the lanes in turn (so that their 16-byte
// accesses to a channel's states and to a token's B and C lie side by side); they add their parts of y by shuffles, in
// a fixed order.  a [inner][N] = -exp(A_log), times log2(e) in the bfloat16 form (`decay_minus_one`).
template <typename T, int SN, int PHASE>
__global__ void __launch_bounds__(SCAN_THREADS)
selective_scan_kernel(T* __restrict__ out, size_t ldo, const T* __restrict__ x, size_t ldx, const float* __restrict__ raw, size_t ldr,
                      const float* __restrict__ a2, const T* __restrict__ B, size_t ldb, const T* __restrict__ C, size_t ldc,
                      const float* __restrict__ Dv, const T* __restrict__ z, size_t ldz, float* __restrict__ state, size_t slot_stride,
                      float* __restrict__ dt_sum, const int32_t* __restrict__ seq_start, const int32_t* __restrict__ seq_slot,
                      int n_seq, int T_rows, int inner, int N, int ln_log2, int vec) {
    extern __shared__ __align__(16) float smem[];
    const int LN = 1 << ln_log2, CH = SCAN_THREADS >> ln_log2, Np = LN * SN;
    float* sB = smem;                                   // [SCAN_TILE][Np]
    float* sC = sB + SCAN_TILE * Np;                    // [SCAN_TILE][Np]
    float* sdt = sC + SCAN_TILE * Np;                   // [SCAN_TILE][CH]
    float* sx = sdt + SCAN_TILE * CH;                   // [SCAN_TILE][CH]
    float* sy = sx + SCAN_TILE * CH;                    // [SCAN_TILE][CH]
    grid_dep_launch();
    grid_dep_wait();
    const int s = blockIdx.x, c0 = blockIdx.y * CH, n_ch = min(CH, inner - c0), tid = threadIdx.x;
    if (PHASE == 0 && s == 0)                           // rows of the packed batch that belong to nobody
        for (int t = seq_start[n_seq]; t < T_rows; ++t)
            for (int c = tid; c < n_ch; c += SCAN_THREADS) out[(size_t)t * ldo + c0 + c] = from_f32<T>(0.f);
    const int slot = seq_slot[s], t0 = seq_start[s], t1 = seq_start[s + 1];
    if (slot < 0) {
        if (PHASE == 0)
            for (int t = t0; t < t1; ++t)
                for (int c = tid; c < n_ch; c += SCAN_THREADS) out[(size_t)t * ldo + c0 + c] = from_f32<T>(0.f);
        return;
    }
    if (t1 <= t0) return;
    const int ch = tid >> ln_log2, l = tid & (LN - 1), c = c0 + ch;
    const bool own = ch < n_ch;
    float* sst = state + (size_t)slot * slot_stride + (size_t)(own ? c : c0) * N;
    const float* arow = a2 + (size_t)(own ? c : c0) * N;
    float S[SN], A[SN];
#pragma unroll
    for (int g = 0; g < SN / 4; ++g) {
        const int n = 4 * (l + (g << ln_log2));
        float4 sv = make_float4(0.f, 0.f, 0.f, 0.f), av = sv;
        if (own && n < N) {
            if (vec) {
                if (PHASE != 1) sv = *reinterpret_cast<const float4*>(sst + n);
                av = *reinterpret_cast<const float4*>(arow + n);
            } else {
                if (PHASE != 1) { sv.x = sst[n]; if (n + 1 < N) sv.y = sst[n + 1]; if (n + 2 < N) sv.z = sst[n + 2]; if (n + 3 < N) sv.w = sst[n + 3]; }
                av.x = arow[n]; if (n + 1 < N) av.y = arow[n + 1]; if (n + 2 < N) av.z = arow[n + 2]; if (n + 3 < N) av.w = arow[n + 3];
            }
        }
        S[4 * g] = sv.x; S[4 * g + 1] = sv.y; S[4 * g + 2] = sv.z; S[4 * g + 3] = sv.w;
        A[4 * g] = av.x; A[4 * g + 1] = av.y; A[4 * g + 2] = av.z; A[4 * g + 3] = av.w;
    }
    const float d_of = own ? Dv[c] : 0.f;
    float sum = 0.f;                                    // PHASE 1: of dt over the chunk
    for (int base = t0; base < t1; base += SCAN_TILE) {
        const int nt = min(SCAN_TILE, t1 - base);
        __syncthreads();
        for (int e = tid; e < SCAN_TILE * Np; e += SCAN_THREADS) {
            const int tt = e / Np, n = e - tt * Np;
            const bool in = tt < nt && n < N;
            sB[e] = in ? to_f32(B[(size_t)(base + tt) * ldb + n]) : 0.f;
            if (PHASE != 1) sC[e] = in ? to_f32(C[(size_t)(base + tt) * ldc + n]) : 0.f;
        }
        for (int e = tid; e < SCAN_TILE * CH; e += SCAN_THREADS) {
            const int tt = e / CH, k = e - tt * CH;
            const bool in = tt < nt && k < n_ch;
            sdt[e] = in ? softplus_f32(raw[(size_t)(base + tt) * ldr + c0 + k]) : 0.f;
            sx[e] = in ? to_f32(x[(size_t)(base + tt) * ldx + c0 + k]) : 0.f;
        }
        __syncthreads();
#pragma unroll 2
        for (int tt = 0; tt < nt; ++tt) {
            const float dt = sdt[tt * CH + ch], xv = sx[tt * CH + ch], u = dt * xv;
            if (PHASE == 1) sum += dt;
            float acc = 0.f;
            const float4* b4 = reinterpret_cast<const float4*>(sB + tt * Np) + l;
            const float4* c4 = reinterpret_cast<const float4*>(sC + tt * Np) + l;
#pragma unroll
            for (int g = 0; g < SN / 4; ++g) {
                const float4 bb = b4[g << ln_log2];
                const float ba[4] = {bb.x, bb.y, bb.z, bb.w};
#pragma unroll
                for (int j = 0; j < 4; ++j)
                    S[4 * g + j] = fmaf(decay_minus_one<T>(dt, A[4 * g + j]), S[4 * g + j], fmaf(u, ba[j], S[4 * g + j]));
                if (PHASE != 1) {
                    const float4 cc = c4[g << ln_log2];
                    acc = fmaf(cc.x, S[4 * g], acc);
                    acc = fmaf(cc.y, S[4 * g + 1], acc);
                    acc = fmaf(cc.z, S[4 * g + 2], acc);
                    acc = fmaf(cc.w, S[4 * g + 3], acc);
                }
            }
            if (PHASE != 1) {
                for (int off = LN >> 1; off > 0; off >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, off);
                if (l == 0) sy[tt * CH + ch] = fmaf(d_of, xv, acc);
            }
        }
        if (PHASE != 1) {
            __syncthreads();
            for (int e = tid; e < nt * CH; e += SCAN_THREADS) {
                const int tt = e / CH, k = e - tt * CH;
                if (k < n_ch) {
                    const size_t row = (size_t)(base + tt);
                    out[row * ldo + c0 + k] = from_f32<T>(sy[e] * silu_f32(to_f32(z[row * ldz + c0 + k])));
                }
            }
        }
    }
    if (PHASE == 1 && own && l == 0) dt_sum[(size_t)slot * inner + c] = sum;
    if (PHASE != 2) {
#pragma unroll
        for (int g = 0; g < SN / 4; ++g) {
            const int n = 4 * (l + (g << ln_log2));
            if (own && n < N) {
                if (vec) *reinterpret_cast<float4*>(sst + n) = make_float4(S[4 * g], S[4 * g + 1], S[4 * g + 2], S[4 * g + 3]);
                else
#pragma unroll
                    for (int j = 0; j < 4; ++j) if (n + j < N) sst[n + j] = S[4 * g + j];
            }
        }
    }
}

// chunk_state[c] (the state chunk c ends with from an empty one) becomes the state it starts from; the slot gets the
// sequence's last state.  One thread per state element (channel, n); a chunk's decay is exp(rate x sum of its `logs`), or a
// power of two (`base2`): `rate` [inner][N] per element, or null for a rate of one (N = 1).
__global__ void channel_prefix_kernel(float* __restrict__ chunk_state, const float* __restrict__ logs, const float* __restrict__ rate,
                                      float* __restrict__ state, size_t slot_stride, const int32_t* __restrict__ seq_chunk,
                                      const int32_t* __restrict__ seq_slot, int inner, int N, int base2) {
    grid_dep_launch();
    grid_dep_wait();
    const int s = blockIdx.x, slot = seq_slot[s], k0 = seq_chunk[s], k1 = seq_chunk[s + 1];
    if (slot < 0 || k1 <= k0) return;
    const size_t n_el = (size_t)inner * N;
    for (size_t e = (size_t)blockIdx.y * blockDim.x + threadIdx.x; e < n_el; e += (size_t)gridDim.y * blockDim.x) {
        const size_t c = e / N;
        const float r = rate ? rate[e] : 1.0f;
        float S = state[(size_t)slot * slot_stride + e];
        for (int k = k0; k < k1; k += AHEAD) {
            float added[AHEAD], lg[AHEAD];
#pragma unroll
            for (int g = 0; g < AHEAD; ++g) {
                added[g] = k + g < k1 ? chunk_state[(size_t)(k + g) * n_el + e] : 0.f;
                lg[g] = k + g < k1 ? logs[(size_t)(k + g) * inner + c] : 0.f;
            }
#pragma unroll
            for (int g = 0; g < AHEAD; ++g)
                if (k + g < k1) {
                    chunk_state[(size_t)(k + g) * n_el + e] = S;
                    S = fmaf(base2 ? exp2f(r * lg[g]) : expf(r * lg[g]), S, added[g]);
                }
        }
        state[(size_t)slot * slot_stride + e] = S;
    }
}

// ----------------------------------------------------------------------------- gated linear recurrent unit

// sigmoid and gelu for a bfloat16 engine on the fast exponential and division (32-bit, off by about 1e-6), else in full.
template <typename T> __device__ __forceinline__ float unit_sigmoid(float v) {
    return sizeof(T) == 2 ? __fdividef(1.0f, 1.0f + __expf(-v)) : sigmoid_f32(v);
}
template <typename T> __device__ __forceinline__ float unit_gelu(float v) { return sizeof(T) == 2 ? gelu_tanh_fast(v) : gelu_tanh(v); }

// A thread per channel.  gates [T][2 n]: per block of `bs` channels the r half, then the i half; bias likewise [2 n];
// rate [n] = 8 softplus(lam).  The tokens' gates and decays do not depend on the state: AHEAD tokens' are taken side by
// side, then the chain.
template <typename T, int PHASE>
__global__ void gated_lru_kernel(T* __restrict__ out, size_t ldo, const T* __restrict__ u, size_t ldu, const float* __restrict__ gates,
                                 size_t ldg, const float* __restrict__ bias, const float* __restrict__ rate, const T* __restrict__ y,
                                 size_t ldy, float* __restrict__ state, size_t slot_stride, float* __restrict__ log_sum,
                                 const int32_t* __restrict__ seq_start, const int32_t* __restrict__ seq_slot, int n_seq, int T_rows,
                                 int n, int bs) {
    grid_dep_launch();
    grid_dep_wait();
    const int s = blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x;
    if (c >= n) return;
    if (PHASE == 0 && s == 0)
        for (int t = seq_start[n_seq]; t < T_rows; ++t) out[(size_t)t * ldo + c] = from_f32<T>(0.f);
    const int slot = seq_slot[s], t0 = seq_start[s], t1 = seq_start[s + 1];
    if (slot < 0) {
        if (PHASE == 0)
            for (int t = t0; t < t1; ++t) out[(size_t)t * ldo + c] = from_f32<T>(0.f);
        return;
    }
    if (t1 <= t0) return;
    const int b = c / bs, at_r = 2 * b * bs + (c - b * bs), at_i = at_r + bs;
    const float br = bias[at_r], bi = bias[at_i], k = rate[c];
    float* mine = state + (size_t)slot * slot_stride + c;
    float S = PHASE == 1 ? 0.f : *mine;
    float logs = 0.f;
    for (int base = t0; base < t1; base += AHEAD) {
        float r[AHEAD], i[AHEAD], uv[AHEAD], yv[AHEAD];
#pragma unroll
        for (int g = 0; g < AHEAD; ++g) {
            const size_t row = (size_t)min(base + g, t1 - 1);
            r[g] = gates[row * ldg + at_r];
            i[g] = gates[row * ldg + at_i];
            uv[g] = to_f32(u[row * ldu + c]);
            if (PHASE != 1) yv[g] = to_f32(y[row * ldy + c]);
        }
#pragma unroll
        for (int g = 0; g < AHEAD; ++g) {
            const float log_a = -k * unit_sigmoid<T>(r[g] + br);
            const float e = expm1f(log_a);              // a - 1; 1 - a^2 = -e (2 + e)
            const float in = sqrtf(-e * (2.0f + e)) * unit_sigmoid<T>(i[g] + bi) * uv[g];
            if (base + g < t1) {
                S = fmaf(e, S, S + in);
                if (PHASE == 1) logs += log_a;
                else out[(size_t)(base + g) * ldo + c] = from_f32<T>(S * unit_gelu<T>(yv[g]));
            }
        }
    }
    if (PHASE == 1) log_sum[(size_t)slot * n + c] = logs;
    if (PHASE != 2) *mine = S;
}

// ----------------------------------------------------------------------------- Mamba-2

// From the step sizes' projection (bias included): dt = softplus(raw), and the decay less one, exp(-exp(A_log_h) dt) - 1.
__global__ void ssd_gates_kernel(float* __restrict__ a, float* __restrict__ dt, const float* __restrict__ raw, size_t ldr,
                                 const float* __restrict__ a_log, int T_rows, int H) {
    grid_dep_launch();
    grid_dep_wait();
    const long long e = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (e >= (long long)T_rows * H) return;
    const int t = (int)(e / H), h = (int)(e - (long long)t * H);
    const float d = softplus_f32(raw[(size_t)t * ldr + h]);
    dt[e] = d;
    a[e] = expm1f(-expf(a_log[h]) * d);
}

// One block per row: v = (o + D_h x) silu(z), kept in shared memory; each of n / part parts divided by its root mean
// square, times w.  A part per warp in turn, or, where there are fewer parts than warps, the block on one after another.
template <typename T>
__global__ void ssd_output_kernel(T* __restrict__ out, size_t ldo, const float* __restrict__ o, size_t ldi, const T* __restrict__ x,
                                  size_t ldx, const T* __restrict__ z, size_t ldz, const float* __restrict__ Dv,
                                  const void* __restrict__ w, int w_dtype, int n, int dv, int part, float eps) {
    extern __shared__ float v_of[];                     // [n], then a reciprocal root per part
    __shared__ float scratch[33];
    float* rstd = v_of + n;
    grid_dep_launch();
    grid_dep_wait();
    const size_t t = blockIdx.x;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5, parts = n / part;
    for (int i = threadIdx.x; i < n; i += blockDim.x)
        v_of[i] = fmaf(Dv[i / dv], to_f32(x[t * ldx + i]), o[t * ldi + i]) * silu_f32(to_f32(z[t * ldz + i]));
    __syncthreads();
    if (parts >= warps) {
        for (int g = warp; g < parts; g += warps) {
            float q = 0.f;
            for (int i = lane; i < part; i += 32) q = fmaf(v_of[g * part + i], v_of[g * part + i], q);
            q = warp_sum(q);
            if (lane == 0) rstd[g] = 1.0f / sqrtf(q / (float)part + eps);
        }
    } else {
        for (int g = 0; g < parts; ++g) {
            float q = 0.f;
            for (int i = threadIdx.x; i < part; i += blockDim.x) q = fmaf(v_of[g * part + i], v_of[g * part + i], q);
            q = block_sum(q, scratch);
            if (threadIdx.x == 0) rstd[g] = 1.0f / sqrtf(q / (float)part + eps);
        }
    }
    __syncthreads();
    for (int i = threadIdx.x; i < n; i += blockDim.x)
        out[t * ldo + i] = from_f32<T>(v_of[i] * rstd[i / part] * load_as_f32(w, w_dtype, i));
}

struct ScanArgs {
    void* out; long long ldo; const void* x; long long ldx; const float* raw; long long ldr; const float* a2; const void* B;
    long long ldb; const void* C; long long ldc; const float* D; const void* z; long long ldz; int T_rows, inner, N;
};

template <typename T, int SN>
int launch_selective(int phase, const ScanArgs& p, float* state, long long slot_stride, float* dt_sum, const int32_t* starts,
                     const int32_t* slots, int n_seq, int ln_log2, cudaStream_t stream) {
    const int CH = SCAN_THREADS >> ln_log2, Np = SN << ln_log2;
    const size_t smem = (size_t)SCAN_TILE * (2 * Np + 3 * CH) * sizeof(float);
    const int vec = p.N % 4 == 0 && slot_stride % 4 == 0 && ((uintptr_t)state % 16) == 0 && ((uintptr_t)p.a2 % 16) == 0;
    const dim3 grid(n_seq, (p.inner + CH - 1) / CH);
    cudaError_t e;
#define GO(PHASE) do { e = smem > 48 * 1024 ? cudaFuncSetAttribute(selective_scan_kernel<T, SN, PHASE>, \
        cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) : cudaSuccess; \
    if (e == cudaSuccess) e = qs_launch_dependent(selective_scan_kernel<T, SN, PHASE>, grid, dim3(SCAN_THREADS), smem, stream, (T*)p.out, \
        (size_t)p.ldo, (const T*)p.x, (size_t)p.ldx, p.raw, (size_t)p.ldr, p.a2, (const T*)p.B, (size_t)p.ldb, (const T*)p.C, \
        (size_t)p.ldc, p.D, (const T*)p.z, (size_t)p.ldz, state, (size_t)slot_stride, dt_sum, starts, slots, n_seq, p.T_rows, p.inner, \
        p.N, ln_log2, vec); } while (0)
    if (phase == 0) GO(0); else if (phase == 1) GO(1); else GO(2);
#undef GO
    if (e != cudaSuccess) return qs_fail(QS_ERR_INTERNAL, "selective_scan: %s", cudaGetErrorString(e));
    return qs_check_launch("selective_scan");
}

int launch_prefix(float* chunk_state, const float* logs, const float* rate, float* state, long long slot_stride,
                  const int32_t* seq_chunk, const int32_t* seq_slot, int n_seq, int inner, int N, int base2, cudaStream_t stream) {
    long long by = ((long long)inner * N + 255) / 256;
    if (by > 1024) by = 1024;
    cudaError_t e = qs_launch_dependent(channel_prefix_kernel, dim3(n_seq, (unsigned)by), dim3(256), 0, stream, chunk_state, logs, rate,
                                        state, (size_t)slot_stride, seq_chunk, seq_slot, inner, N, base2);
    if (e != cudaSuccess) return qs_fail(QS_ERR_INTERNAL, "channel_prefix: %s", cudaGetErrorString(e));
    return qs_check_launch("channel_prefix");
}

}  // namespace

// x [T, C] (row stride ldx, type `dtype`) -> out [T, C]; taps [C][n_taps], bias [C] or null; held [slots][n_taps - 1][C]
// of type `dtype` (null for one tap).  `decode`: every row is one token of its own sequence, and held is updated in
// the same pass; else held is only read (`qs_conv_keep` updates it afterwards).
QS_API int qs_short_conv(void* out, long long ldo, const void* x, long long ldx, int dtype, const void* taps, int w_dtype,
                         const void* bias, int b_dtype, int n_taps, void* held, long long slot_stride, const int32_t* tok_slot,
                         const int32_t* tok_pos, int T_rows, int C, int act, int decode, cudaStream_t stream) {
    if (T_rows == 0) return QS_OK;
    QS_REQUIRE(T_rows > 0 && C > 0 && n_taps >= 1, "short_conv: bad sizes");
    QS_REQUIRE(n_taps == 1 || held, "short_conv: a convolution without its state");
    QS_REQUIRE(dtype == QS_F32 || dtype == QS_BF16, "short_conv: unknown dtype %d", dtype);
    typedef __nv_bfloat16 bf16;
    cudaError_t e;
    if (decode) {
        const dim3 grid(T_rows, (C + 127) / 128);
#define STEP(T) e = qs_launch_dependent(short_conv_step_kernel<T>, grid, dim3(128), 0, stream, (T*)out, (size_t)ldo, (const T*)x, (size_t)ldx, \
        taps, w_dtype, bias, b_dtype, n_taps, (T*)held, (size_t)slot_stride, tok_slot, C, act)
        if (dtype == QS_F32) STEP(float); else STEP(bf16);
#undef STEP
    } else {
        const int unit = dtype == QS_F32 ? 4 : 8;       // elements of 16 bytes
        const bool vec = C % 8 == 0 && ldx % unit == 0 && ldo % unit == 0 && slot_stride % unit == 0 && ((uintptr_t)x % 16) == 0 &&
                         ((uintptr_t)out % 16) == 0 && ((uintptr_t)held % 16) == 0 && ((uintptr_t)taps % 32) == 0 && ((uintptr_t)bias % 32) == 0;
        const int per = vec ? 8 : 1, threads = 128;
        const dim3 grid((T_rows + CONV_TOKENS - 1) / CONV_TOKENS, (C / per + threads) / threads);
#define CONV1(T, V, NT) e = qs_launch_dependent(short_conv_kernel<T, V, NT>, grid, dim3(threads), 0, stream, (T*)out, (size_t)ldo, (const T*)x, (size_t)ldx, \
        taps, w_dtype, bias, b_dtype, n_taps, (const T*)held, (size_t)slot_stride, tok_slot, tok_pos, T_rows, C, act)
#define CONV(T) do { if (!vec) CONV1(T, 1, 0); else if (n_taps == 4) CONV1(T, 8, 4); else if (n_taps == 3) CONV1(T, 8, 3); else if (n_taps == 2) CONV1(T, 8, 2); \
        else CONV1(T, 8, 0); } while (0)
        if (dtype == QS_F32) CONV(float); else CONV(bf16);
#undef CONV
#undef CONV1
    }
    if (e != cudaSuccess) return qs_fail(QS_ERR_INTERNAL, "short_conv: %s", cudaGetErrorString(e));
    return qs_check_launch("short_conv");
}

QS_API int qs_conv_keep(void* held, long long slot_stride, const void* x, long long ldx, int dtype, int C, int n_taps,
                        const int32_t* seq_start, const int32_t* seq_slot, int n_seq, cudaStream_t stream) {
    if (n_seq == 0 || n_taps <= 1) return QS_OK;
    QS_REQUIRE(n_seq > 0 && C > 0 && held, "conv_keep: bad sizes");
    const dim3 grid(n_seq, (C + 127) / 128);
    cudaError_t e;
    if (dtype == QS_F32)
        e = qs_launch_dependent(conv_keep_kernel<float>, grid, dim3(128), 0, stream, (float*)held, (size_t)slot_stride, (const float*)x,
                                (size_t)ldx, C, n_taps, seq_start, seq_slot);
    else if (dtype == QS_BF16)
        e = qs_launch_dependent(conv_keep_kernel<__nv_bfloat16>, grid, dim3(128), 0, stream, (__nv_bfloat16*)held, (size_t)slot_stride,
                                (const __nv_bfloat16*)x, (size_t)ldx, C, n_taps, seq_start, seq_slot);
    else return qs_fail(QS_ERR_INVALID_INPUT, "conv_keep: unknown dtype %d", dtype);
    if (e != cudaSuccess) return qs_fail(QS_ERR_INTERNAL, "conv_keep: %s", cudaGetErrorString(e));
    return qs_check_launch("conv_keep");
}

// x, z [T, inner], B, C [T, N] and out [T, inner] of type `dtype`; raw [T, inner] float32 (the step sizes before the
// softplus, bias included); a2 [inner][N] = -exp(A_log), for bfloat16 times log2(e), D [inner] float32; state [slots][inner][N] float32.
// With `chunk_start` (see qs_state_scan) the chunks run side by side: chunk_state [n_chunks][inner][N] and chunk_logs
// [n_chunks][inner] are scratch.
QS_API int qs_selective_scan(void* out, long long ldo, const void* x, long long ldx, const float* raw, long long ldr, const float* a2,
                             const void* B, long long ldb, const void* C, long long ldc, const float* D, const void* z, long long ldz,
                             int dtype, float* state, long long slot_stride, const int32_t* seq_start, const int32_t* seq_slot,
                             int n_seq, int T_rows, int inner, int N, const int32_t* chunk_start, const int32_t* chunk_ids,
                             int n_chunks, const int32_t* seq_chunk, float* chunk_state, float* chunk_logs, cudaStream_t stream) {
    if (n_seq == 0 || T_rows == 0) return QS_OK;
    QS_REQUIRE(n_seq > 0 && T_rows > 0 && inner > 0 && N > 0, "selective_scan: bad sizes");
    QS_REQUIRE(N <= 512, "selective_scan: %d states per channel above 512", N);
    QS_REQUIRE(dtype == QS_F32 || dtype == QS_BF16, "selective_scan: unknown dtype %d", dtype);
    QS_REQUIRE(!chunk_start || (n_chunks > 0 && chunk_ids && seq_chunk && chunk_state && chunk_logs), "selective_scan: chunks without their scratch");
    // few tokens: few states per lane, many lanes (the state's traffic counts); long walks: fewer shuffles per state.
    // The number of states per lane fixes the order of a channel's sum; it depends on N only.
    const int sn = N <= 128 ? (N > 8 ? 8 : 4) : 16;
    int ln_log2 = 0;
    while ((sn << ln_log2) < N) ++ln_log2;
    const ScanArgs p = {out, ldo, x, ldx, raw, ldr, a2, B, ldb, C, ldc, D, z, ldz, T_rows, inner, N};
#define SCAN1(T, PHASE, STATE, STRIDE, STARTS, SLOTS, NS) (sn == 4 ? launch_selective<T, 4>(PHASE, p, STATE, STRIDE, chunk_logs, STARTS, SLOTS, NS, ln_log2, stream) \
        : sn == 8 ? launch_selective<T, 8>(PHASE, p, STATE, STRIDE, chunk_logs, STARTS, SLOTS, NS, ln_log2, stream) \
                  : launch_selective<T, 16>(PHASE, p, STATE, STRIDE, chunk_logs, STARTS, SLOTS, NS, ln_log2, stream))
#define SCAN(PHASE, STATE, STRIDE, STARTS, SLOTS, NS) (dtype == QS_F32 ? SCAN1(float, PHASE, STATE, STRIDE, STARTS, SLOTS, NS) \
        : SCAN1(__nv_bfloat16, PHASE, STATE, STRIDE, STARTS, SLOTS, NS))
    if (!chunk_start) return SCAN(0, state, slot_stride, seq_start, seq_slot, n_seq);
    const long long per = (long long)inner * N;
    int rc = SCAN(1, chunk_state, per, chunk_start, chunk_ids, n_chunks);
    if (rc == QS_OK) rc = launch_prefix(chunk_state, chunk_logs, a2, state, slot_stride, seq_chunk, seq_slot, n_seq, inner, N, dtype != QS_F32, stream);
    if (rc == QS_OK) rc = SCAN(2, chunk_state, per, chunk_start, chunk_ids, n_chunks);
    return rc;
#undef SCAN
#undef SCAN1
}

// u, y and out [T, n] of type `dtype`; gates [T, 2 n] float32 without bias, per block of `bs` channels (r | i); bias [2 n]
// in the same order, rate [n] = 8 softplus(lam), state [slots][n], all float32.  Chunks as for qs_selective_scan with
// chunk_state [n_chunks][n].
QS_API int qs_gated_lru(void* out, long long ldo, const void* u, long long ldu, const float* gates, long long ldg, const float* bias,
                        const float* rate, const void* y, long long ldy, int dtype, float* state, long long slot_stride,
                        const int32_t* seq_start, const int32_t* seq_slot, int n_seq, int T_rows, int n, int bs,
                        const int32_t* chunk_start, const int32_t* chunk_ids, int n_chunks, const int32_t* seq_chunk,
                        float* chunk_state, float* chunk_logs, cudaStream_t stream) {
    if (n_seq == 0 || T_rows == 0) return QS_OK;
    QS_REQUIRE(n_seq > 0 && T_rows > 0 && n > 0 && bs > 0 && n % bs == 0, "gated_lru: bad sizes");
    QS_REQUIRE(dtype == QS_F32 || dtype == QS_BF16, "gated_lru: unknown dtype %d", dtype);
    QS_REQUIRE(!chunk_start || (n_chunks > 0 && chunk_ids && seq_chunk && chunk_state && chunk_logs), "gated_lru: chunks without their scratch");
    typedef __nv_bfloat16 bf16;
    cudaError_t e = cudaSuccess;
    const int threads = 128;
#define GO1(T, PHASE, STATE, STRIDE, STARTS, SLOTS, NS) e = qs_launch_dependent(gated_lru_kernel<T, PHASE>, dim3(NS, (n + threads - 1) / threads), \
        dim3(threads), 0, stream, (T*)out, (size_t)ldo, (const T*)u, (size_t)ldu, gates, (size_t)ldg, bias, rate, (const T*)y, (size_t)ldy, \
        STATE, (size_t)(STRIDE), chunk_logs, STARTS, SLOTS, NS, T_rows, n, bs)
#define GO(PHASE, STATE, STRIDE, STARTS, SLOTS, NS) do { if (dtype == QS_F32) GO1(float, PHASE, STATE, STRIDE, STARTS, SLOTS, NS); \
        else GO1(bf16, PHASE, STATE, STRIDE, STARTS, SLOTS, NS); } while (0)
    if (!chunk_start) GO(0, state, slot_stride, seq_start, seq_slot, n_seq);
    else {
        GO(1, chunk_state, n, chunk_start, chunk_ids, n_chunks);
        if (e == cudaSuccess) {
            const int rc = launch_prefix(chunk_state, chunk_logs, nullptr, state, slot_stride, seq_chunk, seq_slot, n_seq, n, 1, 0, stream);
            if (rc != QS_OK) return rc;
            GO(2, chunk_state, n, chunk_start, chunk_ids, n_chunks);
        }
    }
#undef GO
#undef GO1
    if (e != cudaSuccess) return qs_fail(QS_ERR_INTERNAL, "gated_lru: %s", cudaGetErrorString(e));
    return qs_check_launch("gated_lru");
}

QS_API int qs_ssd_gates(float* a, float* dt, const float* raw, long long ldr, const float* a_log, int T_rows, int H, cudaStream_t stream) {
    if (T_rows == 0) return QS_OK;
    QS_REQUIRE(T_rows > 0 && H > 0, "ssd_gates: bad sizes");
    const long long total = (long long)T_rows * H;
    cudaError_t e = qs_launch_dependent(ssd_gates_kernel, dim3((unsigned)((total + 127) / 128)), dim3(128), 0, stream, a, dt, raw,
                                        (size_t)ldr, a_log, T_rows, H);
    if (e != cudaSuccess) return qs_fail(QS_ERR_INTERNAL, "ssd_gates: %s", cudaGetErrorString(e));
    return qs_check_launch("ssd_gates");
}

// o [T, n] float32, x, z and out [T, n] of type `dtype`, D [n / dv] float32 (one per head of dv), w [n]; n / parts
// neighbouring elements share a root mean square.
QS_API int qs_ssd_output(void* out, long long ldo, const float* o, long long ldi, const void* x, long long ldx, const void* z,
                         long long ldz, int dtype, const float* D, const void* w, int w_dtype, int rows, int n, int dv, int parts,
                         float eps, cudaStream_t stream) {
    if (rows == 0) return QS_OK;
    QS_REQUIRE(rows > 0 && n > 0 && dv > 0 && n % dv == 0 && parts > 0 && n % parts == 0, "ssd_output: bad sizes n=%d dv=%d parts=%d", n, dv, parts);
    const size_t smem = (size_t)(n + parts) * sizeof(float);
    QS_REQUIRE(smem <= 200 * 1024, "ssd_output: %d channels above the shared memory of a block", n);
    const int threads = n >= 2048 ? 512 : 128;
    cudaError_t e = cudaSuccess;
#define GO(T) do { if (smem > 48 * 1024) e = cudaFuncSetAttribute(ssd_output_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    if (e == cudaSuccess) e = qs_launch_dependent(ssd_output_kernel<T>, dim3(rows), dim3(threads), smem, stream, (T*)out, (size_t)ldo, o, (size_t)ldi, \
        (const T*)x, (size_t)ldx, (const T*)z, (size_t)ldz, D, w, w_dtype, n, dv, n / parts, eps); } while (0)
    if (dtype == QS_F32) GO(float);
    else if (dtype == QS_BF16) GO(__nv_bfloat16);
    else return qs_fail(QS_ERR_INVALID_INPUT, "ssd_output: unknown dtype %d", dtype);
#undef GO
    if (e != cudaSuccess) return qs_fail(QS_ERR_INTERNAL, "ssd_output: %s", cudaGetErrorString(e));
    return qs_check_launch("ssd_output");
}
