// A real-gated linear recurrent unit: a recurrence with a diagonal decay that the input itself sets.
//
// u [T, C] is split into ``blocks`` equal parts of channels; with a square matrix per part and gate,
//     r = sigmoid(R u + r_bias),  i = sigmoid(I u + i_bias),  a = e^(rate_c r)   (rate_c <= 0: a learned number),
//     S <- a S + i u sqrt(1 - a^2),       out = S * gelu(y)   (tanh form; y [T, C] another branch).
// Everything behind the two products' 32-bit sums is 32-bit; S lives in 32-bit rows per sequence, zero at its start.
//
//   gl_unit_gates   both gates' products and what follows from them.  The two matrices' rows alternate (r of channel
//                   c, then i of channel c), so that a thread's neighbouring sums are one channel's gates.  For prompts
//                   it leaves (a, sqrt(1 - a^2) i u) per token and channel; with one token a sequence it makes the
//                   step itself, state row included, and writes out.
//   gl_unit_scan    the recurrence over the tokens of every sequence, and out.
//
// With d = 1 - a = -(e^(log a) - 1) both factors come from one exponential that is exact near zero:
// 1 - a^2 = d (2 - d).
#include "common.cuh"

// FAST: the hardware's exponential, reciprocal and square root, each off by a few 2^-23 of its value.  They enter the
// recurrence as errors of that size in log a and in what is written, which the 16-bit rounding of u outweighs by far;
// the 32-bit path takes the exact forms.
template <bool FAST>
__device__ __forceinline__ float gu_sigmoid(float x) {
    return FAST ? __fdividef(1.0f, 1.0f + __expf(-x)) : 1.0f / (1.0f + expf(-x));
}
template <bool FAST>
__device__ __forceinline__ float gu_sqrt(float x) {
    if (!FAST) return sqrtf(x);
    float y;
    asm("sqrt.approx.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// 1 - e^x for x <= 0: near zero from the series of e^x - 1 to x^9/9! (below 2^-28 here), Horner in 32-bit
template <bool FAST>
__device__ __forceinline__ float gu_one_minus_exp(float x) {
    if (x > -0.5f) {
        float p = 2.755731922e-6f;
        p = fmaf(p, x, 2.48015873e-5f);
        p = fmaf(p, x, 1.984126984e-4f);
        p = fmaf(p, x, 1.388888889e-3f);
        p = fmaf(p, x, 8.333333333e-3f);
        p = fmaf(p, x, 4.166666667e-2f);
        p = fmaf(p, x, 1.666666667e-1f);
        p = fmaf(p, x, 0.5f);
        p = fmaf(p, x, 1.0f);
        return -p * x;
    }
    return 1.0f - (FAST ? __expf(x) : expf(x));
}

struct UnitGatesArgs {
    const void* u;            // [T, C] activation type
    const void* w;            // [blocks, 2 * size, size] weight type: rows r, i of a channel alternate
    const float* bias;        // [2 * C] likewise
    const float* rate;        // [C]: log a = rate * r
    float2* ab;               // [T, C]: a and sqrt(1 - a^2) i u (prompts)
    // one token a sequence (step != 0):
    const void* y;            // activation type, row pitch y_ld, first column y_off
    void* out;                // [T, C] activation type
    float* state;             // [slots, state_stride], S [C] first
    const int* tok_seq;       // [T]
    const int* seq_slot;      // [B]
    int T, C, blocks, y_ld, y_off, state_stride, step;
};

// a channel's gates' sums to its decay and input
template <bool FAST>
__device__ __forceinline__ float2 gu_factors(float rs, float is, float u, float rate) {
    const float d = gu_one_minus_exp<FAST>(rate * gu_sigmoid<FAST>(rs));
    return make_float2(1.0f - d, gu_sqrt<FAST>(d * (2.0f - d)) * gu_sigmoid<FAST>(is) * u);
}

// the other branch's activation, for results rounded to TA
template <typename TA>
__device__ __forceinline__ float gu_gelu(float y) {
    if constexpr (sizeof(TA) == 2) return gl_activate_bf16_grade(y, GL_ACT_GELU_TANH);
    else return gl_activate<true>(y, GL_ACT_GELU_TANH);
}

template <typename TA>
__device__ __forceinline__ void gu_finish(const UnitGatesArgs& g, int t, int c, float rs, float is, float u) {
    const float2 f = gu_factors<sizeof(TA) == 2>(rs + g.bias[2 * c], is + g.bias[2 * c + 1], u, g.rate[c]);
    if (!g.step) {
        g.ab[(size_t)t * g.C + c] = f;
        return;
    }
    float* S = g.state + (size_t)g.seq_slot[g.tok_seq[t]] * g.state_stride + c;
    const float s = fmaf(f.x, *S, f.y);
    *S = s;
    gl_store((TA*)g.out + (size_t)t * g.C + c,
             s * gu_gelu<TA>(gl_load((const TA*)g.y + (size_t)t * g.y_ld + g.y_off + c)));
}

#define GG_BM 64
#define GG_BN 64
#define GG_BK 16

template <typename TA, typename TW>
__global__ void __launch_bounds__(256)
unit_gates_kernel(UnitGatesArgs g) {
    __shared__ float As[GG_BK][GG_BM + 4];
    __shared__ float Ws[GG_BK][GG_BN + 4];
    gl_grid_launch_dependents();
    gl_grid_wait();
    const int size = g.C / g.blocks, N = 2 * size;
    const TA* U = (const TA*)g.u + (size_t)blockIdx.z * size;
    const TW* W = (const TW*)g.w + (size_t)blockIdx.z * N * size;
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const int m0 = blockIdx.y * GG_BM, n0 = blockIdx.x * GG_BN;
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
    for (int k0 = 0; k0 < size; k0 += GG_BK) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int e = tid + i * 256, r = e >> 4, c = e & 15;
            const int k = k0 + c;
            float va = 0.f, vw = 0.f;
            if (k < size) {
                if (m0 + r < g.T) va = gl_load(U + (size_t)(m0 + r) * g.C + k);
                if (n0 + r < N) vw = gl_load(W + (size_t)(n0 + r) * size + k);
            }
            As[c][r] = va;
            Ws[c][r] = vw;
        }
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < GG_BK; ++kk) {
            float av[4], wv[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) av[i] = As[kk][ty * 4 + i];
#pragma unroll
            for (int j = 0; j < 4; ++j) wv[j] = Ws[kk][tx * 4 + j];
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], wv[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int m = m0 + ty * 4 + i;
        if (m >= g.T) continue;
#pragma unroll
        for (int j = 0; j < 4; j += 2) {
            const int n = n0 + tx * 4 + j;
            if (n >= N) continue;
            gu_finish<TA>(g, m, blockIdx.z * size + n / 2, acc[i][j], acc[i][j + 1], gl_load(U + (size_t)m * g.C + n / 2));
        }
    }
}

// The same on the tensor cores for bfloat16 in whole 16-byte pieces: a block takes 64 tokens x 32 channels of a part,
// each of its 4 warps 16 tokens; K passes through shared memory 64 at a time with cp.async, two stages; mma.sync
// m16n8k16 with 32-bit sums, of which a thread's neighbouring two are one channel's gates.
#define GT_ROW (64 * 2 + 16)

__device__ __forceinline__ void gt_cp16(unsigned dst, const void* src, int bytes) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes));
}
__device__ __forceinline__ void gt_ldm4(unsigned addr, unsigned& r0, unsigned& r1, unsigned& r2, unsigned& r3) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void gt_mma(float (&d)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

__global__ void __launch_bounds__(128)
unit_gates_tc_kernel(UnitGatesArgs g) {
    __shared__ __align__(16) unsigned char sA[2][64 * GT_ROW];
    __shared__ __align__(16) unsigned char sW[2][64 * GT_ROW];
    gl_grid_launch_dependents();
    const int size = g.C / g.blocks, N = 2 * size;
    const __nv_bfloat16* U = (const __nv_bfloat16*)g.u + (size_t)blockIdx.z * size;
    const __nv_bfloat16* W = (const __nv_bfloat16*)g.w + (size_t)blockIdx.z * N * size;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, grp = lane >> 2, t = lane & 3;
    const int m0 = blockIdx.y * 64, n0 = blockIdx.x * 64;
    const unsigned a_base[2] = {(unsigned)__cvta_generic_to_shared(sA[0]), (unsigned)__cvta_generic_to_shared(sA[1])};
    const unsigned w_base[2] = {(unsigned)__cvta_generic_to_shared(sW[0]), (unsigned)__cvta_generic_to_shared(sW[1])};
    auto fetch_w = [&](int k0, int st) {
        for (int i = tid; i < 64 * 8; i += 128) {
            const int r = i >> 3, c = i & 7;
            const bool ok = k0 + c * 8 < size && n0 + r < N;
            gt_cp16(w_base[st] + r * GT_ROW + c * 16, ok ? (const void*)(W + (size_t)(n0 + r) * size + k0 + c * 8) : (const void*)W, ok ? 16 : 0);
        }
    };
    auto fetch_a = [&](int k0, int st) {
        for (int i = tid; i < 64 * 8; i += 128) {
            const int r = i >> 3, c = i & 7;
            const bool ok = k0 + c * 8 < size && m0 + r < g.T;
            gt_cp16(a_base[st] + r * GT_ROW + c * 16, ok ? (const void*)(U + (size_t)(m0 + r) * g.C + k0 + c * 8) : (const void*)g.u, ok ? 16 : 0);
        }
    };
    fetch_w(0, 0);                                    // (weights: they come while the kernel before drains)
    gl_grid_wait();
    fetch_a(0, 0);
    asm volatile("cp.async.commit_group;");
    float acc[8][4];
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[j][e] = 0.f;
    const int live_rows = g.T - m0 - warp * 16;       // of this warp's 16
    const int steps = (size + 63) / 64;
    for (int s = 0; s < steps; ++s) {
        const int st = s & 1;
        if (s + 1 < steps) {
            fetch_w((s + 1) * 64, st ^ 1);
            fetch_a((s + 1) * 64, st ^ 1);
        }
        asm volatile("cp.async.commit_group;");
        asm volatile("cp.async.wait_group 1;");
        __syncthreads();
        const int kn = (min(64, size - s * 64) + 15) / 16;        // (what a part has no columns for is zero)
        if (live_rows > 0) {
            for (int kk = 0; kk < kn; ++kk) {
                unsigned af[4];
                gt_ldm4(a_base[st] + (warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * GT_ROW + (kk * 2 + (lane >> 4)) * 16,
                        af[0], af[1], af[2], af[3]);
#pragma unroll
                for (int j = 0; j < 8; j += 2) {
                    unsigned b0, b1, b2, b3;
                    gt_ldm4(w_base[st] + (j * 8 + ((lane >> 4) & 1) * 8 + (lane & 7)) * GT_ROW + (kk * 2 + ((lane >> 3) & 1)) * 16,
                            b0, b1, b2, b3);
                    gt_mma(acc[j], af, b0, b1);
                    gt_mma(acc[j + 1], af, b2, b3);
                }
            }
        }
        __syncthreads();
    }
    asm volatile("cp.async.wait_group 0;");
    // everything the results are made with is asked for before the first is stored: behind a store no load may move up
    const int r_lo = m0 + warp * 16 + grp, c0 = n0 / 2 + t;       // this thread's channels: c0, c0 + 4, ..
    float2 bias[8];
    float rate[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) {
        const bool ok = c0 + 4 * j < size;
        const int cc = blockIdx.z * size + (ok ? c0 + 4 * j : 0);
        bias[j] = *(const float2*)(g.bias + 2 * cc);
        rate[j] = g.rate[cc];
    }
#pragma unroll
    for (int half = 0; half < 2; ++half) {
        const int r = r_lo + 8 * half;
        if (r >= g.T) continue;
        float u[8], s[8], y[8];
        float* S = g.step ? g.state + (size_t)g.seq_slot[g.tok_seq[r]] * g.state_stride + blockIdx.z * size : nullptr;
        const __nv_bfloat16* Y = (const __nv_bfloat16*)g.y + (size_t)r * g.y_ld + g.y_off + blockIdx.z * size;
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            const int c = c0 + 4 * j;
            const bool ok = c < size;
            u[j] = ok ? gl_load(U + (size_t)r * g.C + c) : 0.f;
            s[j] = ok && g.step ? S[c] : 0.f;
            y[j] = ok && g.step ? gl_load(Y + c) : 0.f;
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            const int c = c0 + 4 * j;
            const float2 f = gu_factors<true>(acc[j][2 * half] + bias[j].x, acc[j][2 * half + 1] + bias[j].y, u[j], rate[j]);
            if (c >= size) continue;
            const size_t at = (size_t)r * g.C + blockIdx.z * size + c;
            if (!g.step) {
                g.ab[at] = f;
            } else {
                const float v = fmaf(f.x, s[j], f.y);
                S[c] = v;
                ((__nv_bfloat16*)g.out)[at] = __float2bfloat16_rn(v * gu_gelu<__nv_bfloat16>(y[j]));
            }
        }
    }
}

// The same for prompts, whose tiles are limited by what they fetch: a block takes 128 tokens x 64 channels (128 rows of
// both gates), each of its 8 warps 32 tokens x 32 channels.
#define GW_TILE (128 * GT_ROW)

__global__ void __launch_bounds__(256, 2)
unit_gates_wide_kernel(UnitGatesArgs g) {
    extern __shared__ __align__(16) unsigned char smem[];     // [2] token tiles, [2] weight tiles
    gl_grid_launch_dependents();
    const int size = g.C / g.blocks, N = 2 * size;
    const __nv_bfloat16* U = (const __nv_bfloat16*)g.u + (size_t)blockIdx.z * size;
    const __nv_bfloat16* W = (const __nv_bfloat16*)g.w + (size_t)blockIdx.z * N * size;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, grp = lane >> 2, t = lane & 3;
    const int wm = (warp & 3) * 32, wn = (warp >> 2) * 64;    // this warp's part of the tile
    const int m0 = blockIdx.y * 128, n0 = blockIdx.x * 128;
    const unsigned base = (unsigned)__cvta_generic_to_shared(smem);
    auto fetch = [&](int k0, int st, bool weights) {
        const unsigned dst = base + (weights ? 2 + st : st) * GW_TILE;
        for (int i = tid; i < 128 * 8; i += 256) {
            const int r = i >> 3, c = i & 7;
            const bool ok = k0 + c * 8 < size && (weights ? n0 + r < N : m0 + r < g.T);
            const __nv_bfloat16* src = weights ? W + (size_t)(n0 + r) * size + k0 + c * 8 : U + (size_t)(m0 + r) * g.C + k0 + c * 8;
            gt_cp16(dst + r * GT_ROW + c * 16, ok ? (const void*)src : g.w, ok ? 16 : 0);
        }
    };
    fetch(0, 0, true);                                // (weights: they come while the kernel before drains)
    gl_grid_wait();
    fetch(0, 0, false);
    asm volatile("cp.async.commit_group;");
    float acc[2][8][4];
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 8; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[i][j][e] = 0.f;
    const int steps = (size + 63) / 64;
    for (int s = 0; s < steps; ++s) {
        const int st = s & 1;
        if (s + 1 < steps) {
            fetch((s + 1) * 64, st ^ 1, true);
            fetch((s + 1) * 64, st ^ 1, false);
        }
        asm volatile("cp.async.commit_group;");
        asm volatile("cp.async.wait_group 1;");
        __syncthreads();
        const int kn = (min(64, size - s * 64) + 15) / 16;        // (what a part has no columns for is zero)
        const unsigned sa = base + st * GW_TILE, sw = base + (2 + st) * GW_TILE;
#pragma unroll 1
        for (int kk = 0; kk < kn; ++kk) {
            unsigned af[2][4];
#pragma unroll
            for (int i = 0; i < 2; ++i)
                gt_ldm4(sa + (wm + i * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * GT_ROW + (kk * 2 + (lane >> 4)) * 16,
                        af[i][0], af[i][1], af[i][2], af[i][3]);
#pragma unroll
            for (int j = 0; j < 8; j += 2) {
                unsigned b0, b1, b2, b3;
                gt_ldm4(sw + (wn + j * 8 + ((lane >> 4) & 1) * 8 + (lane & 7)) * GT_ROW + (kk * 2 + ((lane >> 3) & 1)) * 16, b0, b1, b2, b3);
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    gt_mma(acc[i][j], af[i], b0, b1);
                    gt_mma(acc[i][j + 1], af[i], b2, b3);
                }
            }
        }
        __syncthreads();
    }
    asm volatile("cp.async.wait_group 0;");
    const int c0 = (n0 + wn) / 2 + t;                  // this thread's channels: c0, c0 + 4, ..
    float2 bias[8];
    float rate[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) {
        const bool ok = c0 + 4 * j < size;
        const int cc = blockIdx.z * size + (ok ? c0 + 4 * j : 0);
        bias[j] = *(const float2*)(g.bias + 2 * cc);
        rate[j] = g.rate[cc];
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int r = m0 + wm + i * 16 + grp + 8 * half;
            if (r >= g.T) continue;
            float u[8];
#pragma unroll
            for (int j = 0; j < 8; ++j) u[j] = c0 + 4 * j < size ? gl_load(U + (size_t)r * g.C + c0 + 4 * j) : 0.f;
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                const float2 f = gu_factors<true>(acc[i][j][2 * half] + bias[j].x, acc[i][j][2 * half + 1] + bias[j].y, u[j], rate[j]);
                if (c0 + 4 * j < size) g.ab[(size_t)r * g.C + blockIdx.z * size + c0 + 4 * j] = f;
            }
        }
    }
}

GL_API int gl_unit_gates(const UnitGatesArgs* args, int act_dtype, int w_dtype, cudaStream_t stream) {
    const UnitGatesArgs& g = *args;
    if (g.T <= 0) return GL_OK;
    if (g.C <= 0 || g.blocks <= 0 || g.blocks > 65535 || g.C % g.blocks) return GL_ERR_SHAPE;
    if (g.step ? (!g.y || !g.out || !g.state || !g.tok_seq || !g.seq_slot) : !g.ab) return GL_ERR_SHAPE;
    const int size = g.C / g.blocks;
    const dim3 grid((2 * size + GG_BN - 1) / GG_BN, (g.T + GG_BM - 1) / GG_BM, g.blocks);
    if (grid.y > 65535) return GL_ERR_SHAPE;
    const bool pieces = act_dtype == GL_BF16 && w_dtype == GL_BF16 && size % 8 == 0 && !(((uintptr_t)g.u | (uintptr_t)g.w) & 15);
    if (pieces && !g.step && g.T > 64 && size > 32) {
        static bool allowed = false;
        if (!allowed) {
            if (cudaFuncSetAttribute(unit_gates_wide_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 4 * GW_TILE) != cudaSuccess) {
                cudaGetLastError();
                return GL_ERR_SMEM;
            }
            allowed = true;
        }
        return gl_launch(unit_gates_wide_kernel, dim3((2 * size + 127) / 128, (g.T + 127) / 128, g.blocks), dim3(256), 4 * GW_TILE, stream, 1, g);
    }
    if (pieces)
        return gl_launch(unit_gates_tc_kernel, grid, dim3(128), 0, stream, 1, g);
    if (act_dtype == GL_F32 && w_dtype == GL_F32) return gl_launch(unit_gates_kernel<float, float>, grid, dim3(256), 0, stream, 1, g);
    if (act_dtype == GL_BF16 && w_dtype == GL_BF16)
        return gl_launch(unit_gates_kernel<__nv_bfloat16, __nv_bfloat16>, grid, dim3(256), 0, stream, 1, g);
    if (act_dtype == GL_BF16 && w_dtype == GL_F32) return gl_launch(unit_gates_kernel<__nv_bfloat16, float>, grid, dim3(256), 0, stream, 1, g);
    return GL_ERR_DTYPE;
}

// ---------------------------------------------------------------------------
// The recurrence of a prompt.  A block owns 16 channels of one sequence and walks its run in pieces of 128 tokens: 32
// segments of 4 consecutive tokens, a thread a (segment, channel).  A segment is the map S -> P S + Q (P the product
// of its decays, Q its result from zero); a warp a channel puts the 32 maps together in order, and every thread then
// walks its 4 tokens from its segment's start.  The next piece's factors travel while this one is put together.
// ---------------------------------------------------------------------------
#define US_CH 16
#define US_SEG 32
#define US_LEN 4

struct UnitScanArgs {
    const float2* ab;         // [T, C]
    const void* y;            // activation type, row pitch y_ld, first column y_off
    void* out;                // [T, C] activation type
    float* state;             // [slots, state_stride], S [C] first
    const int* seq_slot;
    const int* seq_qstart;
    const int* seq_qlen;
    int B, C, y_ld, y_off, state_stride;
};

template <typename TA>
__global__ void __launch_bounds__(US_CH * US_SEG, 2)
unit_scan_kernel(UnitScanArgs a) {
    __shared__ float sP[US_CH][US_SEG + 1], sQ[US_CH][US_SEG + 1];
    gl_grid_launch_dependents();
    gl_grid_wait();
    const int b = blockIdx.y, ch = threadIdx.x % US_CH, seg = threadIdx.x / US_CH;
    const int c = blockIdx.x * US_CH + ch;
    const bool live = c < a.C;
    const int qlen = a.seq_qlen[b], qstart = a.seq_qstart[b];
    float* state = a.state + (size_t)a.seq_slot[b] * a.state_stride;
    // the warp that puts a channel's segments together keeps the channel's state
    const int w = threadIdx.x >> 5, lane = threadIdx.x & 31, wc = blockIdx.x * US_CH + w;
    float carry = wc < a.C ? state[wc] : 0.f;
    const float2* ab = a.ab + (size_t)qstart * a.C + c;
    const TA* y = (const TA*)a.y + (size_t)qstart * a.y_ld + a.y_off + c;
    TA* out = (TA*)a.out + (size_t)qstart * a.C + c;
    float2 f[US_LEN], nf[US_LEN];
    float yv[US_LEN], ny[US_LEN];
    auto fetch = [&](int s0, float2* ff, float* yy) {
#pragma unroll
        for (int k = 0; k < US_LEN; ++k) {
            const int t = s0 + seg * US_LEN + k;
            const bool ok = live && t < qlen;
            ff[k] = ok ? __ldcg(ab + (size_t)t * a.C) : make_float2(1.f, 0.f);      // a token that does not exist changes nothing
            yy[k] = ok ? gl_load(y + (size_t)t * a.y_ld) : 0.f;
        }
    };
    fetch(0, f, yv);
    for (int s0 = 0; s0 < qlen; s0 += US_SEG * US_LEN) {
        float P = 1.f, Q = 0.f;
#pragma unroll
        for (int k = 0; k < US_LEN; ++k) { P *= f[k].x; Q = fmaf(f[k].x, Q, f[k].y); }
        sP[ch][seg] = P;
        sQ[ch][seg] = Q;
        if (s0 + US_SEG * US_LEN < qlen) fetch(s0 + US_SEG * US_LEN, nf, ny);
        __syncthreads();
        {
            float p = sP[w][lane], q = sQ[w][lane];
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float p0 = __shfl_up_sync(0xffffffffu, p, o), q0 = __shfl_up_sync(0xffffffffu, q, o);
                if (lane >= o) { q = fmaf(p, q0, q); p *= p0; }
            }
            const float end = fmaf(p, carry, q);                     // the state behind this segment
            const float before = __shfl_up_sync(0xffffffffu, end, 1);
            sQ[w][lane] = lane == 0 ? carry : before;
            carry = __shfl_sync(0xffffffffu, end, 31);
        }
        __syncthreads();
        float S = sQ[ch][seg];
#pragma unroll
        for (int k = 0; k < US_LEN; ++k) {
            const int t = s0 + seg * US_LEN + k;
            S = fmaf(f[k].x, S, f[k].y);
            if (live && t < qlen) gl_store(out + (size_t)t * a.C, S * gu_gelu<TA>(yv[k]));
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < US_LEN; ++k) { f[k] = nf[k]; yv[k] = ny[k]; }
    }
    if (lane == 0 && wc < a.C) state[wc] = carry;
}

GL_API int gl_unit_scan(const UnitScanArgs* args, int act_dtype, cudaStream_t stream) {
    const UnitScanArgs& a = *args;
    if (a.B <= 0) return GL_OK;
    if (a.C <= 0 || a.B > 65535 || !a.ab || !a.y || !a.out || !a.state) return GL_ERR_SHAPE;
    const dim3 grid((a.C + US_CH - 1) / US_CH, a.B), block(US_CH * US_SEG);
    if (act_dtype == GL_F32) return gl_launch(unit_scan_kernel<float>, grid, block, 0, stream, 1, a);
    if (act_dtype == GL_BF16) return gl_launch(unit_scan_kernel<__nv_bfloat16>, grid, block, 0, stream, 1, a);
    return GL_ERR_DTYPE;
}
