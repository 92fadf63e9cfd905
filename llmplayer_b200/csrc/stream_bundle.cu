// Hyper-connections: a layer's residual stream is a bundle of S streams per token instead of one. A sublayer with the
// coefficients in[S], out[S], mix[S][S] (indexed [from][to]) reads u = sum_s in[s] x_s through a norm, and its result y
// enters all streams at once:  x'_t = sum_s mix[s][t] x_s + m out[t] y.
//
// One kernel stands between two sublayers. It reads a token's old streams and the finished sublayer's result once,
// writes the new streams once, and on the way forms what comes next: the RMS norm of the next sublayer's
// combination of the NEW streams (in the products' number format), or, behind the last layer, their plain sum. At the
// start all streams equal the embedding's output: the kernel then reads that one row S times over (a stream stride of
// zero), so the copies are never written. A block per token; a thread owns columns, for all streams of the token.
#include "common.cuh"

namespace {

constexpr int BUNDLE_MAX = 32;          // streams at most
// Threads per block: 256 when there are tokens enough to fill the GPU, twice that for a handful of tokens (a decode step,
// where a block's own latency is what counts), if the registers of that many streams allow it.
constexpr int bundle_threads_max(int sx) { return sx > 0 && sx <= 4 ? 512 : 256; }
// At most 64 registers per thread for so few streams, half of the SM's warps resident: what is waited for are the loads, and
// with the compiler's own choice (100 registers, a quarter of the warps) 2,048 rows of 1,024 took 26.6 us instead of 20.5.
constexpr int bundle_blocks_min(int sx) { return sx > 0 && sx <= 4 ? 2 : 1; }

struct BundleArgs {
    const float* src;                   // x: token t's stream s at src + t * src_token + s * src_stream
    long long src_token, src_stream;
    const float* y;                     // the finished sublayer's result [T, d]; null: the streams stay as they are
    const float* mix;                   // [S, S]
    const float* out;                   // [S]
    float scale;                        // m
    float* dst;                         // the new streams [T, S, d]; null: not wanted (behind the last layer)
    const float* in_next;               // [S]: the next sublayer's combination; null: the plain sum
    const float* weight;                // gain [d] of the next norm; null: the combination itself goes to `sum`
    float eps;
    void* normed;                       // [T, d]
    float* sum;                         // [T, d]
    int S, d;
    float* zero;
    long long zero_count;
};

// W values of a row at a time: 4 (rows of a multiple of four values on 16-byte boundaries) or 1
template <int W> struct Piece { float v[W]; };
template <int W> __device__ __forceinline__ Piece<W> load_piece(const float* p) {
    Piece<W> r;
    if constexpr (W == 4) {
        const float4 f = *reinterpret_cast<const float4*>(p);
        r.v[0] = f.x; r.v[1] = f.y; r.v[2] = f.z; r.v[3] = f.w;
    } else {
        r.v[0] = *p;
    }
    return r;
}
template <int W> __device__ __forceinline__ void store_piece(float* p, const Piece<W>& r) {
    if constexpr (W == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
    else *p = r.v[0];
}
template <int W> __device__ __forceinline__ void store_piece(__nv_bfloat16* p, const Piece<W>& r) {
    if constexpr (W == 4) {
        uint2 packed;
        *reinterpret_cast<__nv_bfloat162*>(&packed.x) = __floats2bfloat162_rn(r.v[0], r.v[1]);
        *reinterpret_cast<__nv_bfloat162*>(&packed.y) = __floats2bfloat162_rn(r.v[2], r.v[3]);
        *reinterpret_cast<uint2*>(p) = packed;
    } else {
        *p = __float2bfloat16_rn(r.v[0]);
    }
}

// SX > 0: that many streams, coefficients in registers. SX == 0: a.S streams (at most BUNDLE_MAX), coefficients in shared
// memory and the token's streams read once per new stream.
template <int SX, typename TOUT, int W>
__global__ void __launch_bounds__(bundle_threads_max(SX), bundle_blocks_min(SX))
stream_bundle_kernel(const BundleArgs a) {
    extern __shared__ __align__(16) float u_row[];          // [d]: the combination, until its root mean square is known
    __shared__ float coeff[SX > 0 ? 1 : BUNDLE_MAX * BUNDLE_MAX + 2 * BUNDLE_MAX];
    __shared__ float scratch[32];
    const int S = SX > 0 ? SX : a.S;
    const int tid = threadIdx.x, threads = blockDim.x;
    lp_grid_release();
    constexpr int R = SX > 0 ? SX : 1;
    float mix[R][R], out[R], in[R];
    // weights: nothing that a step writes, so they are read before the wait
    if constexpr (SX > 0) {
#pragma unroll
        for (int s = 0; s < SX; ++s) {
            in[s] = a.in_next ? a.in_next[s] : 1.0f;
            out[s] = a.y ? a.scale * a.out[s] : 0.f;
#pragma unroll
            for (int t = 0; t < SX; ++t) mix[s][t] = a.y ? a.mix[s * SX + t] : 0.f;
        }
    } else {
        for (int i = tid; i < S * S; i += threads) coeff[i] = a.y ? a.mix[i] : 0.f;
        for (int i = tid; i < S; i += threads) {
            coeff[S * S + i] = a.y ? a.scale * a.out[i] : 0.f;
            coeff[S * S + S + i] = a.in_next ? a.in_next[i] : 1.0f;
        }
        __syncthreads();
    }
    lp_grid_wait();
    clear_on_the_side(a.zero, a.zero_count);
    const long long t = blockIdx.x;
    const float* src = a.src + t * a.src_token;
    const float* y = a.y ? a.y + t * a.d : nullptr;
    float* dst = a.dst ? a.dst + t * S * a.d : nullptr;
    const bool norms = a.weight != nullptr;
    float ss = 0.f;
    for (int c = tid * W; c < a.d; c += threads * W) {
        Piece<W> u;
#pragma unroll
        for (int i = 0; i < W; ++i) u.v[i] = 0.f;
        if constexpr (SX > 0) {
            Piece<W> x[SX];
#pragma unroll
            for (int s = 0; s < SX; ++s) x[s] = load_piece<W>(src + s * a.src_stream + c);
            if (y) {
                const Piece<W> yv = load_piece<W>(y + c);
#pragma unroll
                for (int to = 0; to < SX; ++to) {
                    Piece<W> n;
#pragma unroll
                    for (int i = 0; i < W; ++i) {
                        float v = out[to] * yv.v[i];
#pragma unroll
                        for (int s = 0; s < SX; ++s) v = fmaf(mix[s][to], x[s].v[i], v);
                        n.v[i] = v;
                        u.v[i] = fmaf(in[to], v, u.v[i]);
                    }
                    if (dst) store_piece<W>(dst + (long long)to * a.d + c, n);
                }
            } else {
#pragma unroll
                for (int s = 0; s < SX; ++s)
#pragma unroll
                    for (int i = 0; i < W; ++i) u.v[i] = fmaf(in[s], x[s].v[i], u.v[i]);
            }
        } else {
            // any number of streams: the old values of the thread's columns, then every new stream from them
            Piece<W> x[BUNDLE_MAX];
#pragma unroll
            for (int s = 0; s < BUNDLE_MAX; ++s)
                if (s < S) x[s] = load_piece<W>(src + s * a.src_stream + c);
            if (y) {
                const Piece<W> yv = load_piece<W>(y + c);
                for (int to = 0; to < S; ++to) {
                    Piece<W> n;
#pragma unroll
                    for (int i = 0; i < W; ++i) n.v[i] = coeff[S * S + to] * yv.v[i];
#pragma unroll
                    for (int s = 0; s < BUNDLE_MAX; ++s)
                        if (s < S) {
#pragma unroll
                            for (int i = 0; i < W; ++i) n.v[i] = fmaf(coeff[s * S + to], x[s].v[i], n.v[i]);
                        }
#pragma unroll
                    for (int i = 0; i < W; ++i) u.v[i] = fmaf(coeff[S * S + S + to], n.v[i], u.v[i]);
                    if (dst) store_piece<W>(dst + (long long)to * a.d + c, n);
                }
            } else {
#pragma unroll
                for (int s = 0; s < BUNDLE_MAX; ++s)
                    if (s < S) {
#pragma unroll
                        for (int i = 0; i < W; ++i) u.v[i] = fmaf(coeff[S * S + S + s], x[s].v[i], u.v[i]);
                    }
            }
        }
        if (norms) {
            store_piece<W>(u_row + c, u);
#pragma unroll
            for (int i = 0; i < W; ++i) ss = fmaf(u.v[i], u.v[i], ss);
        } else {
            store_piece<W>(a.sum + t * a.d + c, u);
        }
    }
    if (!norms) return;
    const float factor = 1.0f / sqrtf(lp_block_sum(ss, scratch) / (float)a.d + a.eps);
    TOUT* h = reinterpret_cast<TOUT*>(a.normed) + t * a.d;
    for (int c = tid * W; c < a.d; c += threads * W) {          // a thread reads back what it wrote itself
        Piece<W> u = load_piece<W>(u_row + c);
        const Piece<W> g = load_piece<W>(a.weight + c);
#pragma unroll
        for (int i = 0; i < W; ++i) u.v[i] = u.v[i] * factor * g.v[i];
        store_piece<W>(h + c, u);
    }
}

template <typename K> int grant_smem(K kernel, size_t bytes) {
    if (bytes <= 48 * 1024) return 0;
    const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
    if (e != cudaSuccess) {
        snprintf(lp_error_text, sizeof(lp_error_text), "stream_bundle: cannot reserve %zu bytes of shared memory: %s", bytes,
                 cudaGetErrorString(e));
        return (int)e;
    }
    return 0;
}

template <int SX, typename TOUT, int W> int launch_bundle_of(const BundleArgs& a, int T, cudaStream_t stream) {
    const size_t smem = a.weight ? (size_t)a.d * sizeof(float) : 0;
    const int rc = grant_smem(stream_bundle_kernel<SX, TOUT, W>, smem);
    if (rc) return rc;
    const int threads = T <= 2 * lp_sm_count() && a.d > 256 * W ? bundle_threads_max(SX) : 256;
    lp_launch(stream_bundle_kernel<SX, TOUT, W>, (unsigned)T, threads, smem, stream, a);
    return lp_check_launch("stream_bundle");
}
template <int SX, typename TOUT> int launch_bundle(const BundleArgs& a, int T, bool wide, cudaStream_t stream) {
    return wide ? launch_bundle_of<SX, TOUT, 4>(a, T, stream) : launch_bundle_of<SX, TOUT, 1>(a, T, stream);
}

template <typename TOUT> int pick_bundle(const BundleArgs& a, int T, bool wide, cudaStream_t stream) {
    switch (a.S) {
        case 1: return launch_bundle<1, TOUT>(a, T, wide, stream);
        case 2: return launch_bundle<2, TOUT>(a, T, wide, stream);
        case 3: return launch_bundle<3, TOUT>(a, T, wide, stream);
        case 4: return launch_bundle<4, TOUT>(a, T, wide, stream);
        case 8: return launch_bundle<8, TOUT>(a, T, wide, stream);
        default: return launch_bundle<0, TOUT>(a, T, wide, stream);
    }
}

}  // namespace

// src: the streams [T, S, d] (equal == 0) or one row per token that all streams equal, [T, d] (equal != 0). y (optional):
// [T, d], with mix [S, S], out [S], scale; dst (optional): the new streams [T, S, d], may be src. in_next (optional): [S].
// weight (optional) with eps, normed (dtype code): the RMS norm of the combination; without it the combination goes to
// sum [T, d] (which may be src when equal != 0). zero: a float32 buffer cleared on the side.
extern "C" int lp_stream_bundle(const float* src, int equal, const float* y, const float* mix, const float* out, float scale,
                                float* dst, const float* in_next, const float* weight, float eps, void* normed, int normed_dtype,
                                float* sum, int T, int S, int d, float* zero, long long zero_count, cudaStream_t stream) {
    if (T <= 0 || d <= 0) return 0;
    if (S <= 0 || S > BUNDLE_MAX) LP_REFUSE("stream_bundle: %d streams (supported: 1..%d)", S, BUNDLE_MAX);
    if (y && (!mix || !out)) LP_REFUSE("stream_bundle: a result without the coefficients that bring it in");
    if (!y && dst) LP_REFUSE("stream_bundle: new streams without a result that enters them");
    if (weight ? !normed : !sum) LP_REFUSE("stream_bundle: nowhere to write the combination");
    if ((size_t)d * sizeof(float) > 220 * 1024) LP_REFUSE("stream_bundle: rows of %d values", d);
    BundleArgs a{};
    a.src = src;
    a.src_token = equal ? d : (long long)S * d;
    a.src_stream = equal ? 0 : d;
    a.y = y; a.mix = mix; a.out = out; a.scale = scale; a.dst = dst; a.in_next = in_next;
    a.weight = weight; a.eps = eps; a.normed = normed; a.sum = sum; a.S = S; a.d = d;
    a.zero = zero; a.zero_count = zero_count;
    const uintptr_t all = (uintptr_t)src | (uintptr_t)y | (uintptr_t)dst | (uintptr_t)weight | (uintptr_t)sum | (uintptr_t)normed;
    const bool wide = d % 4 == 0 && (all & 15) == 0;
    if (!weight || normed_dtype == LP_F32) return pick_bundle<float>(a, T, wide, stream);
    if (normed_dtype == LP_BF16) return pick_bundle<__nv_bfloat16>(a, T, wide, stream);
    LP_REFUSE("stream_bundle: dtype code %d", normed_dtype);
}
