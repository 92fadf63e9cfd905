// One token per sequence through a recurrent layer, from the projection of the layer's input to the input of its output
// product, in one kernel (the single steps of linear_attention.cu, fused for decode steps). The delta rule:
//
//   short convolutions of the query, key and value channels (the kept inputs move on), silu, unit queries and keys, write
//   strength, decays (one per head, or one per head and key channel from a low-rank map), S <- a S; u = b (v - S^T k);
//   S <- S + k u^T; o = S^T q, the norm of the head's o with its gain, and the output gate (silu or sigmoid; its
//   pre-activations straight from the projection or from a low-rank map).
//
// One CTA per (query / key head, sequence): it forms the head's query and key once and serves every value head that reads
// them, so nothing that one CTA renews (state, kept inputs) is read by another. 16 lanes share a value column's key
// channels (four neighbouring channels per lane and load); the read-outs S^T k and S^T q of a column meet in four shuffles
// and come from the decayed state before the write: o = S^T q + u (k . q). Retention: queries and keys rotated by their
// position, S <- d S + k v^T with a constant d per head, o = S^T q, the norm of the head's o without a gain, the silu gate; a
// CTA per head and sequence. All arithmetic is float32.
#include "common.cuh"

namespace {

constexpr int THREADS = 512;
constexpr int GROUPS = THREADS / 16;        // value columns (times JT) worked on at a time
constexpr int MAX_TAPS = 8;

struct StepArgs {
    const float* proj;         // [B, ld]
    int ld, c_off, b_off, a_off, g_off;    // convolution channels [q | k | v], write strengths, decay and gate columns
    const float* taps;         // [channels, K]
    float* tail;               // [slots, K - 1, channels]
    int K;
    float unit_eps, q_scale;
    const float* dt_bias;      // [H], or [H * dk] with a low-rank map
    const float* a_log;        // [H]
    const void* a_up;          // [H * dk, a_rank] or null
    int a_rank;
    const void* g_up;          // [H * dv, g_rank] or null
    int g_rank;
    int up_bf16, vec;          // number format of the maps; whether their rows can be read 8 values at a time
    int gate_sigmoid;
    const float* gain;         // [dv]
    float norm_eps;
    float* state;              // [slots, H, dv, dk]
    const int* slots;
    int H, G, dk, dv;
    float* zero;
    long long zero_count;
};

__device__ __forceinline__ float softplus(float z) { return z > 20.f ? z : log1pf(expf(z)); }
__device__ __forceinline__ float sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }

// silu of channel c's convolution at this token; the kept inputs move on by one
__device__ __forceinline__ float conv_channel(const StepArgs& a, const float* row, float* kept, int c, int channels) {
    const float x = row[a.c_off + c];
    float hist[MAX_TAPS - 1], w[MAX_TAPS];
#pragma unroll
    for (int j = 0; j < MAX_TAPS - 1; ++j) hist[j] = j < a.K - 1 ? kept[(size_t)j * channels + c] : 0.f;
#pragma unroll
    for (int j = 0; j < MAX_TAPS; ++j) w[j] = j < a.K ? __ldg(a.taps + (size_t)c * a.K + j) : 0.f;
    float acc = 0.f, last = 0.f;
#pragma unroll
    for (int j = 0; j < MAX_TAPS - 1; ++j)
        if (j < a.K - 1) {
            acc = fmaf(w[j], hist[j], acc);
            kept[(size_t)j * channels + c] = j + 1 < a.K - 1 ? hist[j + 1 < MAX_TAPS - 1 ? j + 1 : j] : x;
        }
#pragma unroll
    for (int j = 0; j < MAX_TAPS; ++j) last = j == a.K - 1 ? w[j] : last;
    acc = fmaf(last, x, acc);
    return acc / (1.0f + expf(-acc));
}

// this lane's quarter of up[row] . low
template <typename TW>
__device__ __forceinline__ float quarter_dot(const TW* up, const float* low, int rank, int vec, int sub) {
    float acc = 0.f;
    if (vec) {
        for (int k = sub * 8; k < rank; k += 32) {
            float w[8];
            if (sizeof(TW) == 2) {
                const uint4 raw = __ldg(reinterpret_cast<const uint4*>(up + k));
                const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const float2 f = __bfloat1622float2(p[i]);
                    w[2 * i] = f.x;
                    w[2 * i + 1] = f.y;
                }
            } else {
                const float4 lo = __ldg(reinterpret_cast<const float4*>(up + k)), hi = __ldg(reinterpret_cast<const float4*>(up + k) + 1);
                w[0] = lo.x; w[1] = lo.y; w[2] = lo.z; w[3] = lo.w;
                w[4] = hi.x; w[5] = hi.y; w[6] = hi.z; w[7] = hi.w;
            }
#pragma unroll
            for (int i = 0; i < 8; ++i) acc = fmaf(w[i], low[k + i], acc);
        }
    } else {
        for (int k = sub; k < rank; k += 4) acc = fmaf(lp_to_float(up[k]), low[k], acc);
    }
    return acc;
}

// The state entries of the lane's channels 64 u + 4 l16 + e of JT neighbouring columns from column j0 on.
template <int KPT, int JT>
__device__ __forceinline__ void load_columns(float (*s)[KPT], const float* S, int j0, int l16, int dk, int dv) {
    const bool quads = (dk & 3) == 0;
#pragma unroll
    for (int jj = 0; jj < JT; ++jj) {
        const int j = j0 + jj;
#pragma unroll
        for (int u = 0; u < KPT / 4; ++u) {
            const int c = 64 * u + 4 * l16;
            if (quads) {
                float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
                if (j < dv && c < dk) v = *reinterpret_cast<const float4*>(S + (size_t)j * dk + c);
                s[jj][4 * u] = v.x; s[jj][4 * u + 1] = v.y; s[jj][4 * u + 2] = v.z; s[jj][4 * u + 3] = v.w;
            } else {
#pragma unroll
                for (int e = 0; e < 4; ++e) s[jj][4 * u + e] = (j < dv && c + e < dk) ? S[(size_t)j * dk + c + e] : 0.f;
            }
        }
    }
}
template <int KPT, int JT>
__device__ __forceinline__ void store_columns(const float (*s)[KPT], float* S, int j0, int l16, int dk, int dv) {
    const bool quads = (dk & 3) == 0;
#pragma unroll
    for (int jj = 0; jj < JT; ++jj) {
        const int j = j0 + jj;
#pragma unroll
        for (int u = 0; u < KPT / 4; ++u) {
            const int c = 64 * u + 4 * l16;
            if (j >= dv || c >= dk) continue;
            if (quads)
                *reinterpret_cast<float4*>(S + (size_t)j * dk + c) = make_float4(s[jj][4 * u], s[jj][4 * u + 1], s[jj][4 * u + 2], s[jj][4 * u + 3]);
            else {
#pragma unroll
                for (int e = 0; e < 4; ++e)
                    if (c + e < dk) S[(size_t)j * dk + c + e] = s[jj][4 * u + e];
            }
        }
    }
}

// TW: number format of the low-rank maps. KPT: key channels per lane (dk <= 16 KPT), JT: neighbouring value columns per 16 lanes.
template <typename TW, int KPT, int JT, typename TOut>
__global__ void __launch_bounds__(THREADS)
delta_step_kernel(const StepArgs a, TOut* __restrict__ out) {
    extern __shared__ float sm[];
    const int dk = a.dk, dv = a.dv, R = a.H / a.G;
    float* q_s = sm;                    // [dk]
    float* k_s = q_s + dk;              // [dk]
    float* d_s = k_s + dk;              // [dk] decays
    float* v_s = d_s + dk;              // [dv]
    float* o_s = v_s + dv;              // [dv]
    float* g_s = o_s + dv;              // [dv] gate pre-activations
    float* low_a = g_s + dv;            // [a_rank]
    float* low_g = low_a + (a.a_up ? a.a_rank : 0);
    const int g = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, lane = tid & 31;
    lp_grid_release();
    lp_grid_wait();
    clear_on_the_side(a.zero, a.zero_count);
    const float* row = a.proj + (size_t)b * a.ld;
    const int qk = a.G * dk, channels = 2 * qk + a.H * dv;
    float* kept = a.tail + (size_t)a.slots[b] * (a.K - 1) * channels;
    const int l16 = tid & 15, grp = tid >> 4;

    float s[JT][KPT];                   // requested ahead of what they meet
    auto load = [&](int h, int base) {
        load_columns<KPT, JT>(s, a.state + ((size_t)a.slots[b] * a.H + h) * dv * dk, base + grp * JT, l16, dk, dv);
    };
    load(g * R, 0);
    if (a.a_up)
        for (int i = tid; i < a.a_rank; i += THREADS) low_a[i] = row[a.a_off + i];
    if (a.g_up)
        for (int i = tid; i < a.g_rank; i += THREADS) low_g[i] = row[a.g_off + i];
    for (int i = tid; i < 2 * dk; i += THREADS) {
        const int c = i < dk ? i : i - dk;
        (i < dk ? q_s : k_s)[c] = conv_channel(a, row, kept, (i < dk ? 0 : qk) + g * dk + c, channels);
    }
    __syncthreads();
    // every warp forms the sums over the head's channels for itself
    float qq = 0.f, kk = 0.f, kq = 0.f;
    for (int c = lane; c < dk; c += 32) {
        const float q = q_s[c], k = k_s[c];
        qq = fmaf(q, q, qq);
        kk = fmaf(k, k, kk);
        kq = fmaf(k, q, kq);
    }
    qq = lp_warp_sum(qq);
    kk = lp_warp_sum(kk);
    kq = lp_warp_sum(kq);
    const float fq = a.q_scale / sqrtf(qq + a.unit_eps), fk = 1.0f / sqrtf(kk + a.unit_eps);
    kq *= fq * fk;

    for (int r = 0; r < R; ++r) {
        const int h = g * R + r;
        for (int j = tid; j < dv; j += THREADS) {
            v_s[j] = conv_channel(a, row, kept, 2 * qk + h * dv + j, channels);
            if (!a.g_up) g_s[j] = row[a.g_off + h * dv + j];
        }
        const float rate = expf(a.a_log[h]);
        if (a.a_up || a.g_up) {
            // low-rank maps: four lanes per row, decays' rows first
            const int rows_a = a.a_up ? dk : 0, rows = rows_a + (a.g_up ? dv : 0);
            const int sub = tid & 3;
            for (int i0 = 0; i0 < rows; i0 += THREADS / 4) {
                const int i = i0 + (tid >> 2);
                float z = 0.f;
                if (i < rows_a) z = quarter_dot((const TW*)a.a_up + ((size_t)h * dk + i) * a.a_rank, low_a, a.a_rank, a.vec, sub);
                else if (i < rows) z = quarter_dot((const TW*)a.g_up + ((size_t)h * dv + i - rows_a) * a.g_rank, low_g, a.g_rank, a.vec, sub);
                z += __shfl_xor_sync(0xffffffffu, z, 1);
                z += __shfl_xor_sync(0xffffffffu, z, 2);
                if (sub == 0 && i < rows) {
                    if (i < rows_a) d_s[i] = expf(-rate * softplus(z + a.dt_bias[(size_t)h * dk + i]));
                    else g_s[i - rows_a] = z;
                }
            }
        }
        if (!a.a_up) {
            const float d = expf(-rate * softplus(row[a.a_off + h] + a.dt_bias[h]));
            for (int c = tid; c < dk; c += THREADS) d_s[c] = d;
        }
        const float beta = sigmoid(row[a.b_off + h]);
        __syncthreads();
        float* S = a.state + ((size_t)a.slots[b] * a.H + h) * dv * dk;
        for (int base = 0; base < dv; base += GROUPS * JT) {
            float r1[JT], r2[JT];
#pragma unroll
            for (int jj = 0; jj < JT; ++jj) r1[jj] = r2[jj] = 0.f;
#pragma unroll
            for (int u = 0; u < KPT; ++u) {
                const int c = 64 * (u >> 2) + 4 * l16 + (u & 3);
                const float d = c < dk ? d_s[c] : 0.f, k = c < dk ? k_s[c] * fk : 0.f, q = c < dk ? q_s[c] * fq : 0.f;
#pragma unroll
                for (int jj = 0; jj < JT; ++jj) {
                    s[jj][u] *= d;
                    r1[jj] = fmaf(s[jj][u], k, r1[jj]);
                    r2[jj] = fmaf(s[jj][u], q, r2[jj]);
                }
            }
#pragma unroll
            for (int o = 1; o < 16; o <<= 1)
#pragma unroll
                for (int jj = 0; jj < JT; ++jj) {
                    r1[jj] += __shfl_xor_sync(0xffffffffu, r1[jj], o);
                    r2[jj] += __shfl_xor_sync(0xffffffffu, r2[jj], o);
                }
#pragma unroll
            for (int jj = 0; jj < JT; ++jj) {
                const int j = base + grp * JT + jj;
                const float w = j < dv ? beta * (v_s[j] - r1[jj]) : 0.f;
                if (l16 == 0 && j < dv) o_s[j] = fmaf(w, kq, r2[jj]);
                r1[jj] = w * fk;                  // k is unit only with this factor
            }
#pragma unroll
            for (int u = 0; u < KPT; ++u) {
                const int c = 64 * (u >> 2) + 4 * l16 + (u & 3);
                const float k = c < dk ? k_s[c] : 0.f;
#pragma unroll
                for (int jj = 0; jj < JT; ++jj) s[jj][u] = fmaf(k, r1[jj], s[jj][u]);
            }
            store_columns<KPT, JT>(s, S, base + grp * JT, l16, dk, dv);
            if (base + GROUPS * JT < dv) load(h, base + GROUPS * JT);
            else if (r + 1 < R) load(h + 1, 0);
        }
        __syncthreads();
        float ss = 0.f;
        for (int j = lane; j < dv; j += 32) ss = fmaf(o_s[j], o_s[j], ss);
        ss = lp_warp_sum(ss);
        const float f = 1.0f / sqrtf(ss / (float)dv + a.norm_eps);
        for (int j = tid; j < dv; j += THREADS) {
            const float z = g_s[j];
            const float act = a.gate_sigmoid ? sigmoid(z) : z * sigmoid(z);
            out[((size_t)b * a.H + h) * dv + j] = lp_from_float<TOut>(o_s[j] * f * a.gain[j] * act);
        }
        __syncthreads();               // v, o, the gates and the decays are free for the next head
    }
}


// ---------------------------------------------------------------- retention
struct RetentionArgs {
    const float* proj;         // [B, ld]: queries, keys [H, dk], values, gate [H, dv]
    int ld, q_off, k_off, v_off, g_off;
    const float* inv_freq;     // [rd / 2] or null
    int rd, interleaved;
    const int* positions;      // [B]
    const float* decays;       // [H]
    float q_scale, norm_eps;
    float* state;              // [slots, H, dv, dk]
    const int* slots;
    int H, dk, dv;
    float* zero;
    long long zero_count;
};

template <int KPT, int JT, typename TOut>
__global__ void __launch_bounds__(THREADS)
retention_step_kernel(const RetentionArgs a, TOut* __restrict__ out) {
    extern __shared__ float sm[];
    const int dk = a.dk, dv = a.dv;
    float* q_s = sm;                    // [dk]
    float* k_s = q_s + dk;              // [dk]
    float* v_s = k_s + dk;              // [dv]
    float* o_s = v_s + dv;              // [dv]
    const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, lane = tid & 31;
    lp_grid_release();
    lp_grid_wait();
    clear_on_the_side(a.zero, a.zero_count);
    const int l16 = tid & 15, grp = tid >> 4;
    const float* row = a.proj + (size_t)b * a.ld;
    float* S = a.state + ((size_t)a.slots[b] * a.H + h) * dv * dk;
    float s[JT][KPT];
    load_columns<KPT, JT>(s, S, grp * JT, l16, dk, dv);
    for (int i = tid; i < 2 * dk; i += THREADS) {
        const int c = i < dk ? i : i - dk;
        const float* head = row + (i < dk ? a.q_off : a.k_off) + h * dk;
        float val = head[c];
        if (c < a.rd) {
            const int half = a.rd >> 1;
            const bool first = a.interleaved ? (c & 1) == 0 : c < half;
            const int pair = a.interleaved ? c >> 1 : (first ? c : c - half);
            const float other = head[a.interleaved ? (c ^ 1) : (first ? c + half : c - half)];
            float sn, cs;
            sincosf((float)a.positions[b] * a.inv_freq[pair], &sn, &cs);
            val = first ? val * cs - other * sn : val * cs + other * sn;
        }
        (i < dk ? q_s : k_s)[c] = i < dk ? val * a.q_scale : val;
    }
    for (int j = tid; j < dv; j += THREADS) v_s[j] = row[a.v_off + h * dv + j];
    __syncthreads();
    const float d = a.decays[h];
    for (int base = 0; base < dv; base += GROUPS * JT) {
        const int j0 = base + grp * JT;
        float v[JT], r[JT];
#pragma unroll
        for (int jj = 0; jj < JT; ++jj) {
            v[jj] = j0 + jj < dv ? v_s[j0 + jj] : 0.f;
            r[jj] = 0.f;
        }
#pragma unroll
        for (int u = 0; u < KPT; ++u) {
            const int c = 64 * (u >> 2) + 4 * l16 + (u & 3);
            const float k = c < dk ? k_s[c] : 0.f, q = c < dk ? q_s[c] : 0.f;
#pragma unroll
            for (int jj = 0; jj < JT; ++jj) {
                s[jj][u] = fmaf(d, s[jj][u], k * v[jj]);
                r[jj] = fmaf(s[jj][u], q, r[jj]);
            }
        }
        store_columns<KPT, JT>(s, S, j0, l16, dk, dv);
        if (base + GROUPS * JT < dv) load_columns<KPT, JT>(s, S, j0 + GROUPS * JT, l16, dk, dv);
#pragma unroll
        for (int o = 1; o < 16; o <<= 1)
#pragma unroll
            for (int jj = 0; jj < JT; ++jj) r[jj] += __shfl_xor_sync(0xffffffffu, r[jj], o);
#pragma unroll
        for (int jj = 0; jj < JT; ++jj)
            if (l16 == 0 && j0 + jj < dv) o_s[j0 + jj] = r[jj];
    }
    __syncthreads();
    float ss = 0.f;
    for (int j = lane; j < dv; j += 32) ss = fmaf(o_s[j], o_s[j], ss);
    ss = lp_warp_sum(ss);
    const float f = 1.0f / sqrtf(ss / (float)dv + a.norm_eps);
    for (int j = tid; j < dv; j += THREADS) {
        const float z = row[a.g_off + h * dv + j];
        out[((size_t)b * a.H + h) * dv + j] = lp_from_float<TOut>(o_s[j] * f * (z * sigmoid(z)));
    }
}

}  // namespace

// One new token for each of B sequences through a retention. proj: float32 [B, ld] (see RetentionArgs for the columns); positions:
// int32 [B]; out: [B, H * dv] float32 or bfloat16.
extern "C" int lp_retention_step(const float* proj, int ld, int q_off, int k_off, int v_off, int g_off, const float* inv_freq, int rd,
                                 int interleaved, const int* positions, const float* decays, float q_scale, float norm_eps, float* state,
                                 const int* slots, void* out, int out_dtype, int B, int H, int dk, int dv, float* zero,
                                 long long zero_count, cudaStream_t stream) {
    if (B <= 0) return 0;
    if (H <= 0 || H > 65535 || B > 65535 || dk <= 0 || dk > 512 || dv <= 0) LP_REFUSE("retention_step: %d sequences, %d heads of %d x %d", B, H, dk, dv);
    if (q_off < 0 || k_off < 0 || v_off < 0 || g_off < 0 || q_off + H * dk > ld || k_off + H * dk > ld || v_off + H * dv > ld || g_off + H * dv > ld)
        LP_REFUSE("retention_step: columns at %d, %d, %d, %d do not fit rows of %d", q_off, k_off, v_off, g_off, ld);
    if (rd < 0 || rd > dk || (rd & 1) || (rd > 0 && !inv_freq)) LP_REFUSE("retention_step: a rotation over %d of %d channels", rd, dk);
    if (((uintptr_t)state & 15) != 0) LP_REFUSE("retention_step: the state must be aligned to 16 bytes");
    const RetentionArgs a{proj, ld, q_off, k_off, v_off, g_off, inv_freq, rd, interleaved, positions, decays, q_scale, norm_eps, state, slots,
                          H, dk, dv, zero, zero_count};
    const size_t smem = ((size_t)2 * dk + 2 * dv) * sizeof(float);
    if (smem > 46 * 1024) LP_REFUSE("retention_step: heads of %d x %d do not fit shared memory", dk, dv);
    const dim3 grid(H, B);
#define LP_RSTEP(KPT, JT)                                                                                                      \
    do {                                                                                                                       \
        if (out_dtype == LP_BF16) lp_launch(retention_step_kernel<KPT, JT, __nv_bfloat16>, grid, THREADS, smem, stream, a, (__nv_bfloat16*)out); \
        else if (out_dtype == LP_F32) lp_launch(retention_step_kernel<KPT, JT, float>, grid, THREADS, smem, stream, a, (float*)out); \
        else LP_REFUSE("retention_step: output dtype code %d", out_dtype);                                                     \
    } while (0)
    if (dk <= 64) LP_RSTEP(4, 4);
    else if (dk <= 128) LP_RSTEP(8, 4);
    else if (dk <= 256) LP_RSTEP(16, 2);
    else LP_RSTEP(32, 1);
#undef LP_RSTEP
    return lp_check_launch("retention_step");
}

// One new token for each of B sequences through a delta rule. proj: float32 [B, ld] (see StepArgs for the columns); out: [B, H * dv] float32 or
// bfloat16. a_up / g_up null: one decay per head, gate pre-activations straight from the projection.
extern "C" int lp_delta_step(const float* proj, int ld, int c_off, int b_off, int a_off, int g_off, const float* taps, float* tail,
                             int K, float unit_eps, float q_scale, const float* dt_bias, const float* a_log, const void* a_up,
                             int a_rank, const void* g_up, int g_rank, int up_dtype, int gate_sigmoid, const float* gain, float norm_eps,
                             float* state, const int* slots, void* out, int out_dtype, int B, int H, int G, int dk, int dv,
                             float* zero, long long zero_count, cudaStream_t stream) {
    if (B <= 0) return 0;
    if (H <= 0 || G <= 0 || H % G || dk <= 0 || dk > 512 || dv <= 0) LP_REFUSE("delta_step: %d heads on %d of %d x %d", H, G, dk, dv);
    if (K < 1 || K > MAX_TAPS) LP_REFUSE("delta_step: %d taps (supported: 1..%d)", K, MAX_TAPS);
    if (G > 65535 || B > 65535) LP_REFUSE("delta_step: %d heads x %d sequences exceed the grid", G, B);
    const int channels = 2 * G * dk + H * dv;
    if (c_off < 0 || c_off + channels > ld || b_off < 0 || b_off + H > ld || a_off < 0 || a_off + (a_up ? a_rank : H) > ld || g_off < 0 ||
        g_off + (g_up ? g_rank : H * dv) > ld)
        LP_REFUSE("delta_step: columns at %d, %d, %d, %d do not fit rows of %d", c_off, b_off, a_off, g_off, ld);
    if ((a_up && a_rank <= 0) || (g_up && g_rank <= 0)) LP_REFUSE("delta_step: factors of %d and %d values", a_rank, g_rank);
    if (up_dtype != LP_F32 && up_dtype != LP_BF16) LP_REFUSE("delta_step: dtype code %d of the maps", up_dtype);
    if (((uintptr_t)state & 15) != 0) LP_REFUSE("delta_step: the state must be aligned to 16 bytes");
    StepArgs a{proj, ld, c_off, b_off, a_off, g_off, taps, tail, K, unit_eps, q_scale, dt_bias, a_log, a_up, a_up ? a_rank : 0, g_up,
               g_up ? g_rank : 0, up_dtype == LP_BF16, 0, gate_sigmoid, gain, norm_eps, state, slots, H, G, dk, dv, zero, zero_count};
    a.vec = a.a_rank % 8 == 0 && a.g_rank % 8 == 0 && (((uintptr_t)a_up | (uintptr_t)g_up) & 15) == 0;
    const size_t smem = ((size_t)3 * dk + 3 * dv + a.a_rank + a.g_rank) * sizeof(float);
    if (smem > 46 * 1024) LP_REFUSE("delta_step: %d x %d with factors of %d and %d do not fit shared memory", dk, dv, a_rank, g_rank);
    const dim3 grid(G, B);
#define LP_STEP(TW, KPT, JT)                                                                                                   \
    do {                                                                                                                       \
        if (out_dtype == LP_BF16) lp_launch(delta_step_kernel<TW, KPT, JT, __nv_bfloat16>, grid, THREADS, smem, stream, a, (__nv_bfloat16*)out); \
        else if (out_dtype == LP_F32) lp_launch(delta_step_kernel<TW, KPT, JT, float>, grid, THREADS, smem, stream, a, (float*)out); \
        else LP_REFUSE("delta_step: output dtype code %d", out_dtype);                                                         \
    } while (0)
#define LP_STEP_SIZE(TW)                                                                                                       \
    do {                                                                                                                       \
        if (dk <= 64) LP_STEP(TW, 4, 4);                                                                                       \
        else if (dk <= 128) LP_STEP(TW, 8, 4);                                                                                 \
        else if (dk <= 256) LP_STEP(TW, 16, 2);                                                                                \
        else LP_STEP(TW, 32, 1);                                                                                               \
    } while (0)
    if (up_dtype == LP_BF16) LP_STEP_SIZE(__nv_bfloat16);
    else LP_STEP_SIZE(float);
#undef LP_STEP_SIZE
#undef LP_STEP
    return lp_check_launch("delta_step");
}
