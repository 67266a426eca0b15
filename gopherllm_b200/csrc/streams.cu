// Several residual streams instead of one (hyper-connections).
//
// A token's residual is a matrix X of S rows of W numbers, 32-bit.  With vectors i, o of S numbers and a matrix M [S, S] a
// sublayer is
//     u = X^T i,      y = sublayer(norm(u)),      X <- M^T X + o y^T:
// row s of M says where the old stream s goes, o how much of y every stream takes.
// Between two sublayers stands one kernel that does both and the norm of the next sublayer's input: it takes y (or
// two branches of a sublayer with a factor each, y = f a + f2 b), updates the streams in place and leaves
// rms(u) * gamma of the new streams in the activation type.  Without y it only reads (before the first layer; behind
// the last one, with i all ones, for selected rows); without ``in_share`` it only updates.
// A block a token; the row u stays in shared memory between the sum of its squares and its use.
#include "common.cuh"

#define ST_MAX_STREAMS 16
#define ST_MAX_THREADS 512

struct StreamArgs {
    float* x;                 // [T, S, W]
    const float* a;           // [T, W] or null: what the sublayer returned
    const float* b;           // [T, W] or null: its second branch
    const float* mix;         // [S, S]: M
    const float* out_share;   // [S]: o
    const float* in_share;    // [S] or null: the next sublayer's i (null: nothing is read)
    const float* gamma;       // [W] or null: no norm, u itself
    void* h;                  // [R, W]
    const int* rows;          // [R] or null: rows of x that are read (without an update)
    int R, S, W;
    float fa, fb, eps;
};

template <int VEC> struct StVec { float v[VEC]; };
template <int VEC>
__device__ __forceinline__ StVec<VEC> st_load(const float* p) {
    StVec<VEC> r;
    if constexpr (VEC == 4) {
        const float4 f = __ldcg((const float4*)p);
        r.v[0] = f.x; r.v[1] = f.y; r.v[2] = f.z; r.v[3] = f.w;
    } else {
        r.v[0] = __ldcg(p);
    }
    return r;
}

// NS: streams the registers hold (S of them in use)
template <typename TO, int NS, int VEC>
__global__ void __launch_bounds__(ST_MAX_THREADS, NS <= 4 ? 2 : 1)
streams_kernel(StreamArgs a) {
    extern __shared__ __align__(16) float row[];          // [W]: u
    __shared__ float ws[ST_MAX_STREAMS * (ST_MAX_STREAMS + 2)];      // mix, out, in
    __shared__ float red[ST_MAX_THREADS / 32];
    gl_grid_launch_dependents();
    const int S = a.S, W = a.W;
    // (weights: they come while the kernel before drains)
    for (int i = threadIdx.x; i < NS * (NS + 2); i += blockDim.x) {
        const int s = i / (NS + 2), k = i - s * (NS + 2);
        float w = 0.f;
        if (s < S) {
            if (k < NS) { if (k < S && a.mix) w = a.mix[s * S + k]; }
            else if (k == NS) { if (a.out_share) w = a.out_share[s]; }
            else if (a.in_share) w = a.in_share[s];
        }
        ws[i] = w;
    }
    gl_grid_wait();
    const int r = blockIdx.x;
    float* x = a.x + (size_t)(a.rows ? a.rows[r] : r) * S * W;
    __syncthreads();
    float wr[NS <= 4 ? NS * (NS + 2) : 1];
    if constexpr (NS <= 4) {
#pragma unroll
        for (int i = 0; i < NS * (NS + 2); ++i) wr[i] = ws[i];
    }
    auto weight = [&](int s, int k) -> float {
        if constexpr (NS <= 4) return wr[s * (NS + 2) + k];
        else return ws[s * (NS + 2) + k];
    };
    float sq = 0.f;
    for (int d = threadIdx.x * VEC; d < W; d += blockDim.x * VEC) {
        StVec<VEC> old[NS];
#pragma unroll
        for (int s = 0; s < NS; ++s)
            if (s < S) old[s] = st_load<VEC>(x + (size_t)s * W + d);
        if (a.a) {
            StVec<VEC> y = st_load<VEC>(a.a + (size_t)r * W + d);
#pragma unroll
            for (int e = 0; e < VEC; ++e) y.v[e] *= a.fa;
            if (a.b) {
                const StVec<VEC> z = st_load<VEC>(a.b + (size_t)r * W + d);
#pragma unroll
                for (int e = 0; e < VEC; ++e) y.v[e] = fmaf(a.fb, z.v[e], y.v[e]);
            }
            StVec<VEC> u;
#pragma unroll
            for (int e = 0; e < VEC; ++e) u.v[e] = 0.f;
#pragma unroll
            for (int t = 0; t < NS; ++t) {
                if (t < S) {
                    StVec<VEC> n;
                    const float o = weight(t, NS), in = weight(t, NS + 1);
#pragma unroll
                    for (int e = 0; e < VEC; ++e) {
                        float v = o * y.v[e];
#pragma unroll
                        for (int s = 0; s < NS; ++s)
                            if (s < S) v = fmaf(weight(s, t), old[s].v[e], v);
                        n.v[e] = v;
                        u.v[e] = fmaf(in, v, u.v[e]);
                    }
                    if constexpr (VEC == 4) *(float4*)(x + (size_t)t * W + d) = make_float4(n.v[0], n.v[1], n.v[2], n.v[3]);
                    else x[(size_t)t * W + d] = n.v[0];
                }
            }
#pragma unroll
            for (int e = 0; e < VEC; ++e) { row[d + e] = u.v[e]; sq = fmaf(u.v[e], u.v[e], sq); }
        } else {
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
                float u = 0.f;
#pragma unroll
                for (int s = 0; s < NS; ++s)
                    if (s < S) u = fmaf(weight(s, NS + 1), old[s].v[e], u);
                row[d + e] = u;
                sq = fmaf(u, u, sq);
            }
        }
    }
    if (!a.in_share) return;
    float inv = 1.0f;
    if (a.gamma) {
        sq = gl_warp_sum(sq);
        if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = sq;
        __syncthreads();
        float tot = 0.f;
        for (int i = 0; i < (int)(blockDim.x >> 5); ++i) tot += red[i];          // same order in every thread
        inv = 1.0f / sqrtf(tot / (float)W + a.eps);
    }
    TO* h = (TO*)a.h + (size_t)r * W;
    for (int d = threadIdx.x * VEC; d < W; d += blockDim.x * VEC) {               // (a thread reads what it wrote)
        float v[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[e] = a.gamma ? row[d + e] * inv * a.gamma[d + e] : row[d + e];
        if constexpr (VEC == 4 && sizeof(TO) == 4) {
            *(float4*)(h + d) = make_float4(v[0], v[1], v[2], v[3]);
        } else if constexpr (VEC == 4) {
            const __nv_bfloat162 p0 = __floats2bfloat162_rn(v[0], v[1]), p1 = __floats2bfloat162_rn(v[2], v[3]);
            uint2 pk;
            pk.x = *(const unsigned*)&p0; pk.y = *(const unsigned*)&p1;
            *(uint2*)(h + d) = pk;
        } else {
            gl_store(h + d, v[0]);
        }
    }
}

template <typename TO, int NS>
static int launch_streams(const StreamArgs& a, cudaStream_t stream) {
    const bool vec = a.W % 4 == 0 && !(((uintptr_t)a.x | (uintptr_t)a.a | (uintptr_t)a.b | (uintptr_t)a.h | (uintptr_t)a.gamma) & 15);
    const size_t smem = (size_t)a.W * sizeof(float);
    const int work = vec ? a.W / 4 : a.W;
    const int threads = work > 256 ? (a.R <= 296 && work > 384 ? 512 : 256) : (work > 128 ? 256 : (work > 64 ? 128 : 64));
    if (vec) return gl_launch(streams_kernel<TO, NS, 4>, dim3((unsigned)a.R), dim3(threads), smem, stream, 1, a);
    return gl_launch(streams_kernel<TO, NS, 1>, dim3((unsigned)a.R), dim3(threads), smem, stream, 1, a);
}

template <typename TO>
static int dispatch_streams(const StreamArgs& a, cudaStream_t stream) {
    if (a.S == 1) return launch_streams<TO, 1>(a, stream);
    if (a.S == 2) return launch_streams<TO, 2>(a, stream);
    if (a.S <= 4) return launch_streams<TO, 4>(a, stream);
    if (a.S <= 8) return launch_streams<TO, 8>(a, stream);
    return launch_streams<TO, ST_MAX_STREAMS>(a, stream);
}

GL_API int gl_streams(const StreamArgs* args, int out_dtype, cudaStream_t stream) {
    const StreamArgs& a = *args;
    if (a.R <= 0) return GL_OK;
    if (a.S <= 0 || a.S > ST_MAX_STREAMS || a.W <= 0 || !a.x) return GL_ERR_SHAPE;
    if (a.a && (!a.mix || !a.out_share || a.rows)) return GL_ERR_SHAPE;
    if ((a.in_share && !a.h) || (!a.in_share && !a.a) || (a.b && !a.a)) return GL_ERR_SHAPE;
    if ((size_t)a.W * sizeof(float) > 40 * 1024) return GL_ERR_SMEM;
    if (out_dtype == GL_F32) return dispatch_streams<float>(a, stream);
    if (out_dtype == GL_BF16) return dispatch_streams<__nv_bfloat16>(a, stream);
    return GL_ERR_DTYPE;
}
