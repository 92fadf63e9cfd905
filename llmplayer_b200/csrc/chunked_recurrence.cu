// Linear-attention recurrences over prompts in chunks of 32 tokens, with the sums inside and between chunks as matrix
// products (the recurrences of linear_attention.cu for steps with many tokens; the same state, the same results up to
// rounding):
//
//     plain:       S_t = diag(a_t) S_(t-1) + k_t v_t^T                                                o_t = S_t^T q_t
//     delta rule:  S <- diag(a_t) S;  u_t = b_t (v_t - S^T k_t);  S <- S + k_t u_t^T                  o_t = S^T q_t
//
// With S the state that enters a chunk, P_i the product of the decays of tokens 1 .. i of the chunk (a vector over the key
// channels) and P_(j,i] that of tokens j + 1 .. i,
//
//     A_ij = sum_c k_ic k_jc P_(j,i],c  (j < i)          B_ij = sum_c q_ic k_jc P_(j,i],c  (j <= i)
//     (I + diag(b) A) U = diag(b) (V - (P k) S),  so  U = U0 - W S  with U0, W the solutions for diag(b) V and diag(b) (P k)
//     o_i = (P_i q_i)^T S + sum_j B_ij u_j               S' = P_32 S + sum_j (P_(j,32] k_j) u_j^T
//
// (the plain recurrence has U = V). Decays enter as running products only, forwards or backwards from a token or a block
// border, so nothing is divided by a product of decays and no logarithm is taken: strong decays (down to zero) are exact.
//
//   prepare   one CTA per (chunk, head, sequence): products of decays, A and B (16 x 16 blocks: between two blocks as sums
//             over factored decays, inside a block with the decays multiplied token by token), the triangular solve with a
//             thread per column, all in float32 arithmetic; the results go to a record per chunk and head, laid out as the
//             operand fragments of the second kernel's products.
//   carry     one CTA per (16 value columns, head, sequence) walks the sequence's chunks in order; the state's columns stay in
//             shared memory. The products run on the tensor cores (mma.sync m16n8k8) at float32 precision: every
//             operand is split into two TF32 parts, x = hi + lo with 22 bits of mantissa together, and hi hi + hi lo + lo hi
//             are summed in float32. Records come by cp.async, one chunk ahead.
#include "common.cuh"

namespace {

constexpr int CT = 32;                  // tokens per chunk
constexpr int HB = 16;                  // tokens per block inside a chunk
constexpr int NC = 16;                  // value columns per CTA of the second kernel
constexpr int THREADS = 256;            // of the first kernel
constexpr int CARRY_THREADS = 512;      // of the second: 16 warps, one per 16 key channels
constexpr int MAX_DK = 256;
constexpr size_t MAX_SMEM = 227 * 1024;

constexpr int DECAY_CHANNEL = 0, DECAY_HEAD = 1, DECAY_FIXED = 2;

// Floats of a record: [W][Q][K^T][B][P_32], fragments of 16 x 8 values each (128 floats: a lane's four values together).
__host__ __device__ __forceinline__ int padded(int dk) { return (dk + 15) / 16 * 16; }
__host__ __device__ __forceinline__ int record_floats(int dkp, bool delta) { return CT * dkp * (delta ? 3 : 2) + CT * CT + dkp; }
__host__ __device__ __forceinline__ int value_floats(int dv) { return (dv + NC - 1) / NC * NC * CT; }

// where element (r, c) of a matrix with `ksteps` = columns / 8 lies in its fragment order (m16n8k8, row operand)
__device__ __forceinline__ int fragment_at(int r, int c, int ksteps) {
    const int lane = (r & 7) * 4 + (c & 3), reg = ((r >> 3) & 1) + ((c >> 2) & 1) * 2;
    return (((r >> 4) * ksteps + (c >> 3)) * 32 + lane) * 4 + reg;
}

__device__ __forceinline__ float rotated_channel(const float* head, int c, int rd, int interleaved, const float2* cs) {
    const float val = __ldg(head + c);
    if (c >= rd) return val;
    const int half = rd >> 1;
    const bool first = interleaved ? (c & 1) == 0 : c < half;
    const int pair = interleaved ? c >> 1 : (first ? c : c - half);
    const float other = __ldg(head + (interleaved ? (c ^ 1) : (first ? c + half : c - half)));
    const float2 a = __ldg(cs + pair);
    return first ? val * a.x - other * a.y : val * a.x + other * a.y;
}

struct Inputs {
    const float* proj;            // [T, ld]: queries at q_off, keys at k_off ([qk heads, dk]), values at v_off ([H, dv])
    int ld, q_off, k_off, v_off;
    const float* decay;           // by `decay_form`: [T, H * dk], [T, H] or [H]
    int decay_form;
    const float* key_gain;        // [T, H] or null
    const float* beta;            // [T, H] or null: the delta rule
    const float2* angles;         // [T, rd / 2] or null
    int rd, interleaved;
    float q_scale;
    int H, dk, dv, qk_group;
};

// ---------------------------------------------------------------- prepare
// PER: key channels per lane of a sum over a head's channels (16 lanes): dk <= 16 PER.
template <int PER>
__global__ void __launch_bounds__(THREADS, PER <= 8 ? 2 : 1)
prepare_kernel(Inputs in, const int* __restrict__ q_start, int first_chunk, int chunks, float* __restrict__ records,
               float* __restrict__ values) {
    extern __shared__ float sm[];
    const int dk = in.dk, dv = in.dv, H = in.H, dkp = padded(dk), ks = dkp + 4;      // rows padded against bank conflicts
    float* qs = sm;                        // [CT][ks]
    float* kk = qs + CT * ks;              // [CT][ks]
    float* gs = kk + CT * ks;              // [CT][ks]
    float* kf = gs + CT * ks;              // [HB][ks]: keys of the second block times the decays since its start
    float* qf = kf + HB * ks;              // [HB][ks]: its queries likewise
    float* ke = qf + HB * ks;              // [HB][ks]: keys of the first block times the decays up to its end
    float* L = ke + HB * ks;               // [CT][CT]: b_i A_ij
    float* Bm = L + CT * CT;               // [CT][CT]
    float* bs = Bm + CT * CT;              // [CT]
    lp_grid_release();
    lp_grid_wait();
    const int h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x;
    const int t0 = q_start[b] + (first_chunk + blockIdx.x) * CT, t1 = q_start[b + 1];
    if (t0 >= t1) return;
    const int n = min(CT, t1 - t0);
    const bool delta = in.beta != nullptr;
    const size_t slot = ((size_t)b * chunks + blockIdx.x) * H + h;
    float* rec = records + slot * record_floats(dkp, delta);
    float* val = values + slot * value_floats(dv);
    float* rec_w = rec;
    float* rec_q = rec + (delta ? CT * dkp : 0);
    float* rec_k = rec_q + CT * dkp;
    float* rec_b = rec_k + CT * dkp;
    float* rec_p = rec_b + CT * CT;
    const int hq = h / in.qk_group;
    // four elements per thread and turn, so that their loads are in flight together
    for (int e0 = tid; e0 < CT * dkp; e0 += 4 * THREADS) {
        float q[4], k[4], g[4];
        int at[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const int e = e0 + u * THREADS;
            const int i = e / dkp, c = e - i * dkp;
            at[u] = e < CT * dkp ? i * ks + c : -1;
            q[u] = k[u] = 0.f;
            g[u] = 1.f;
            if (i < n && c < dk) {
                const float* row = in.proj + (size_t)(t0 + i) * in.ld;
                const float* qh = row + in.q_off + hq * dk;
                const float* kh = row + in.k_off + hq * dk;
                if (in.rd > 0) {
                    const float2* cs = in.angles + (size_t)(t0 + i) * (in.rd >> 1);
                    q[u] = rotated_channel(qh, c, in.rd, in.interleaved, cs);
                    k[u] = rotated_channel(kh, c, in.rd, in.interleaved, cs);
                } else {
                    q[u] = __ldg(qh + c);
                    k[u] = __ldg(kh + c);
                }
                g[u] = in.decay_form == DECAY_FIXED ? __ldg(in.decay + h)
                       : in.decay_form == DECAY_HEAD ? __ldg(in.decay + (size_t)(t0 + i) * H + h)
                                                     : __ldg(in.decay + ((size_t)(t0 + i) * H + h) * dk + c);
                if (in.key_gain) k[u] *= __ldg(in.key_gain + (size_t)(t0 + i) * H + h);
            }
        }
#pragma unroll
        for (int u = 0; u < 4; ++u)
            if (at[u] >= 0) {
                qs[at[u]] = q[u] * in.q_scale;
                kk[at[u]] = k[u];
                gs[at[u]] = g[u];
            }
    }
    for (int i = tid; i < CT; i += THREADS) bs[i] = delta && i < n ? in.beta[(size_t)(t0 + i) * H + h] : 0.f;
    for (int e = tid; e < CT * CT; e += THREADS) L[e] = Bm[e] = 0.f;
    __syncthreads();

    // products of decays, a thread per key channel (forwards; its column of diag(b) (P k) stays in registers for the solve) and
    // one backwards (other threads where there are enough)
    float col[CT];
    const int back = dkp <= THREADS / 2 ? THREADS / 2 : 0;
    if (tid < dkp) {
        const int c = tid;
        float p = 1.f, pb = 1.f;
#pragma unroll
        for (int i = 0; i < CT; ++i) {
            const float g = gs[i * ks + c], k = kk[i * ks + c], q = qs[i * ks + c];
            p *= g;
            rec_q[fragment_at(i, c, dkp >> 3)] = q * p;
            col[i] = bs[i] * k * p;
            if (i >= HB) {
                pb *= g;
                kf[(i - HB) * ks + c] = k * pb;
                qf[(i - HB) * ks + c] = q * pb;
            }
        }
        rec_p[c] = p;
    }
    if (tid >= back && tid - back < dkp) {
        const int c = tid - back;
        float p = 1.f, pb = 1.f;
#pragma unroll
        for (int i = CT - 1; i >= 0; --i) {
            const float g = gs[i * ks + c], k = kk[i * ks + c];
            rec_k[fragment_at(c, i, CT >> 3)] = k * p;
            p *= g;
            if (i < HB) {
                ke[i * ks + c] = k * pb;
                pb *= g;
            }
        }
    }
    __syncthreads();

    // inside the two blocks: thread (block, two neighbouring keys j, 16 lanes over the channels); m = k_j times the decays
    // of tokens j + 1 .. i moves on with i, and the four sums of a row meet in five shuffles
    {
        const int block = tid >> 7, jg = (tid >> 4) & 7, lane = tid & 15;
        const int base = block * HB, j0 = jg * 2;
        float m0[PER], m1[PER];
#pragma unroll
        for (int u = 0; u < PER; ++u) {
            const int c = lane + 16 * u;
            m0[u] = c < dkp ? kk[(base + j0) * ks + c] : 0.f;
            m1[u] = c < dkp ? kk[(base + j0 + 1) * ks + c] : 0.f;
        }
        const int from = (jg & ~1) * 2;            // the two key groups of a warp walk the same rows (shuffles need both)
        for (int i = from; i < HB; ++i) {
            float a0 = 0.f, a1 = 0.f, b0 = 0.f, b1 = 0.f;
            const bool on0 = i > j0, on1 = i > j0 + 1;
#pragma unroll
            for (int u = 0; u < PER; ++u) {
                const int c = lane + 16 * u;
                if (16 * u < dkp) {
                    const float g = gs[(base + i) * ks + c], k = kk[(base + i) * ks + c], q = qs[(base + i) * ks + c];
                    if (on0) m0[u] *= g;
                    if (on1) m1[u] *= g;
                    a0 = fmaf(k, m0[u], a0); b0 = fmaf(q, m0[u], b0);
                    a1 = fmaf(k, m1[u], a1); b1 = fmaf(q, m1[u], b1);
                }
            }
            // lanes 0-7 keep (a0, b0), lanes 8-15 (a1, b1); then each half of those keeps one of the two
            const bool hi8 = lane & 8, hi4 = lane & 4;
            float x = hi8 ? a1 : a0, y = hi8 ? b1 : b0;
            x += __shfl_xor_sync(0xffffffffu, hi8 ? a0 : a1, 8);
            y += __shfl_xor_sync(0xffffffffu, hi8 ? b0 : b1, 8);
            float z = hi4 ? y : x;
            z += __shfl_xor_sync(0xffffffffu, hi4 ? x : y, 4);
            z += __shfl_xor_sync(0xffffffffu, z, 2);
            z += __shfl_xor_sync(0xffffffffu, z, 1);
            const int j = j0 + (hi8 ? 1 : 0);
            if ((lane & 3) == 0) {
                if (hi4) { if (i >= j) Bm[(base + i) * CT + base + j] = z; }
                else if (i > j) L[(base + i) * CT + base + j] = bs[base + i] * z;
            }
        }
    }
    // between the blocks: thread (row of the second, key of the first)
    {
        const int i = tid >> 4, j = tid & 15;
        float a = 0.f, bsum = 0.f;
        const float4* kr = reinterpret_cast<const float4*>(kf + i * ks);
        const float4* qr = reinterpret_cast<const float4*>(qf + i * ks);
        const float4* er = reinterpret_cast<const float4*>(ke + j * ks);
        for (int c = 0; c < dkp >> 2; ++c) {
            const float4 k = kr[c], q = qr[c], e = er[c];
            a = fmaf(k.x, e.x, fmaf(k.y, e.y, fmaf(k.z, e.z, fmaf(k.w, e.w, a))));
            bsum = fmaf(q.x, e.x, fmaf(q.y, e.y, fmaf(q.z, e.z, fmaf(q.w, e.w, bsum))));
        }
        L[(HB + i) * CT + j] = bs[HB + i] * a;
        Bm[(HB + i) * CT + j] = bsum;
    }
    __syncthreads();
    for (int e = tid; e < CT * CT; e += THREADS) rec_b[fragment_at(e / CT, e % CT, CT >> 3)] = Bm[e];

    // the solve: x_i = r_i - sum_(j<i) L_ij x_j, a thread per column of [diag(b) (P k) | diag(b) V]
    const int columns = dkp + (dv + NC - 1) / NC * NC;
    for (int item = tid; item < columns; item += THREADS) {
        const bool key = item < dkp;
        if (key && !delta) continue;
        const int c = item - dkp;
        if (!key) {
#pragma unroll
            for (int i = 0; i < CT; ++i) {
                const float v = (i < n && c < dv) ? __ldg(in.proj + (size_t)(t0 + i) * in.ld + in.v_off + h * dv + c) : 0.f;
                col[i] = delta ? bs[i] * v : v;
            }
        }
        if (delta) {
#pragma unroll
            for (int i = 1; i < CT; ++i) {
                float acc = col[i];
#pragma unroll
                for (int j = 0; j < i; j += 4) {
                    const float4 l = *reinterpret_cast<const float4*>(L + i * CT + j);      // zero from the diagonal on
                    acc = fmaf(-l.x, col[j], acc);
                    if (j + 1 < i) acc = fmaf(-l.y, col[j + 1], acc);
                    if (j + 2 < i) acc = fmaf(-l.z, col[j + 2], acc);
                    if (j + 3 < i) acc = fmaf(-l.w, col[j + 3], acc);
                }
                col[i] = acc;
            }
        }
        if (key) {
#pragma unroll
            for (int i = 0; i < CT; ++i) rec_w[fragment_at(i, item, dkp >> 3)] = col[i];
        } else {
            float* at = val + (c / NC) * (CT * NC) + c % NC;
#pragma unroll
            for (int i = 0; i < CT; ++i) at[i * NC] = col[i];
        }
    }
}

// ---------------------------------------------------------------- carry
// x = hi + lo with two TF32 values: hi is x with its last 13 bits cut off, lo the remainder rounded to TF32 (by integer
// operations: the conversion instruction runs at a fraction of their rate)
__device__ __forceinline__ void split_tf32(float x, uint32_t& hi, uint32_t& lo) {
    hi = __float_as_uint(x) & 0xffffe000u;
    lo = (__float_as_uint(x - __uint_as_float(hi)) + 0x1000u) & 0xffffe000u;
}
__device__ __forceinline__ void mma_tf32(float* c, const uint32_t* a, const uint32_t* b) {
    asm volatile(
        "mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
        : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
}
__device__ __forceinline__ void cp16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

constexpr int SROW = 24;                // floats per row of S and U in shared memory: 16 columns, operand reads without conflicts

// acc[two tiles of 16 x 8] += A[16 x 8 (s1 - s0)] X[8 (s1 - s0) x 16] for the steps s0 .. s1 - 1 of 8 columns of A (in fragment
// order), X split into `xh` + `xl` (rows of SROW); three chains of sums per tile
__device__ __forceinline__ void product(float (*acc)[3][4], const float* frag, const uint32_t* xh, const uint32_t* xl, int s0, int s1,
                                        int lane) {
    const float4* a = reinterpret_cast<const float4*>(frag) + lane;
    const int at = (lane & 3) * SROW + (lane >> 2);
#pragma unroll 4
    for (int s = s0; s < s1; ++s) {
        const float4 av = a[s * 32];
        uint32_t ah[4], al[4];
        split_tf32(av.x, ah[0], al[0]);
        split_tf32(av.y, ah[1], al[1]);
        split_tf32(av.z, ah[2], al[2]);
        split_tf32(av.w, ah[3], al[3]);
#pragma unroll
        for (int w = 0; w < 2; ++w) {
            const int e = at + s * 8 * SROW + w * 8;
            const uint32_t bh[2] = {xh[e], xh[e + 4 * SROW]}, bl[2] = {xl[e], xl[e + 4 * SROW]};
            mma_tf32(acc[w][0], ah, bh);
            mma_tf32(acc[w][1], ah, bl);
            mma_tf32(acc[w][2], al, bh);
        }
    }
}
__device__ __forceinline__ float4 chains(const float (*acc)[4]) {
    return make_float4(acc[0][0] + (acc[1][0] + acc[2][0]), acc[0][1] + (acc[1][1] + acc[2][1]), acc[0][2] + (acc[1][2] + acc[2][2]),
                       acc[0][3] + (acc[1][3] + acc[2][3]));
}

// 16 warps. W S and Q S (32 x 16 each) share the warps, four per 16 rows with a quarter of the key channels each (without W,
// eight per 16 rows of Q S); their parts meet in shared memory. Then warp m owns the state's key channels 16 m .. 16 m + 15:
// its threads hold those entries in registers, shared memory holds them split for the products.
// STAGES: records in flight (two, or one where two do not fit shared memory).
template <int STAGES>
__global__ void __launch_bounds__(CARRY_THREADS)
carry_kernel(float* __restrict__ state, const int* __restrict__ slots, const int* __restrict__ q_start, int first_chunk, int chunks,
             const float* __restrict__ records, const float* __restrict__ values, float* __restrict__ out, int H, int dk, int dv,
             int delta) {
    extern __shared__ float sm[];
    const int dkp = padded(dk), rec_n = record_floats(dkp, delta != 0);
    uint32_t* Sh = reinterpret_cast<uint32_t*>(sm);      // [dkp][SROW] twice: the two parts of S
    uint32_t* Sl = Sh + dkp * SROW;
    uint32_t* Uh = Sl + dkp * SROW;                      // [CT][SROW] twice
    uint32_t* Ul = Uh + CT * SROW;
    float4* parts = reinterpret_cast<float4*>(Ul + CT * SROW);           // [16 warps][2 tiles][32 lanes]
    float4* qs = parts + 16 * 64;                                        // [2][2 tiles][32]: Q S
    float* ring = reinterpret_cast<float*>(qs + 128);    // STAGES records, each followed by the chunk's 32 x 16 values
    const int stage = rec_n + CT * NC;
    lp_grid_release();
    lp_grid_wait();
    const int h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int j0 = blockIdx.x * NC;
    const int begin = q_start[b] + first_chunk * CT, t1 = q_start[b + 1];
    if (begin >= t1) return;
    const int used = min(chunks, (t1 - begin + CT - 1) / CT);
    float* row = state + ((size_t)slots[b] * H + h) * dv * dk;

    auto request = [&](int p) {                     // chunk p's record and values into stage p % STAGES
        if (p < used) {
            const size_t slot = ((size_t)b * chunks + p) * H + h;
            const float* src = records + slot * rec_n;
            const float* val = values + slot * value_floats(dv) + blockIdx.x * (CT * NC);
            float* dst = ring + (p % STAGES) * stage;
            for (int e = tid; e < rec_n / 4; e += CARRY_THREADS) cp16(dst + 4 * e, src + 4 * e);
            for (int e = tid; e < CT * NC / 4; e += CARRY_THREADS) cp16(dst + rec_n + 4 * e, val + 4 * e);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
#pragma unroll
    for (int p = 0; p < STAGES; ++p) request(p);
    const int g8 = lane >> 2, t4 = lane & 3;
    const int kt = dkp >> 4, ks = dkp >> 3;
    const bool owns = warp < kt;
    float s[2][4];
#pragma unroll
    for (int w = 0; w < 2; ++w)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int r = warp * 16 + g8 + (e >> 1) * 8, c = w * 8 + t4 * 2 + (e & 1);
            s[w][e] = (owns && j0 + c < dv && r < dk) ? row[(size_t)(j0 + c) * dk + r] : 0.f;
            if (owns) split_tf32(s[w][e], Sh[r * SROW + c], Sl[r * SROW + c]);
        }
    // this warp's share of the first products: rows 16 mt of W (role 0) or Q (role 1), steps s0 .. s1 over the key channels
    const int nk = delta ? 4 : 8, per = (ks + nk - 1) / nk;
    const int role = delta ? warp >> 3 : 1, mt = delta ? (warp >> 2) & 1 : warp >> 3;
    const int s0 = (warp & (nk - 1)) * per, s1 = min(ks, s0 + per);
    for (int p = 0; p < used; ++p) {
        asm volatile("cp.async.wait_group %0;" ::"n"(STAGES - 1) : "memory");
        __syncthreads();                            // the record is there, and S as the previous chunk left it
        const float* rec = ring + (p % STAGES) * stage;
        const float* rec_q = rec + (delta ? CT * dkp : 0);
        const float* rec_k = rec_q + CT * dkp;
        const float* rec_b = rec_k + CT * dkp;
        const float* rec_p = rec_b + CT * CT;
        const float* val = rec + rec_n;
        {
            float acc[2][3][4] = {};
            product(acc, (role == 1 ? rec_q : rec) + mt * ks * 128, Sh, Sl, s0, s1, lane);
            parts[warp * 64 + lane] = chains(acc[0]);
            parts[warp * 64 + 32 + lane] = chains(acc[1]);
        }
        __syncthreads();
        if (tid < 256) {                            // thread (product, row half, tile, lane): the parts added, in order
            const int what = tid >> 7, half = (tid >> 6) & 1, w = (tid >> 5) & 1;
            float4 sum = make_float4(0.f, 0.f, 0.f, 0.f);
            if (what == 1 || delta) {
                const float4* at = parts + (delta ? what * 8 + half * 4 : half * 8) * 64 + w * 32 + lane;
                for (int k = 0; k < nk; ++k) {
                    const float4 v = at[k * 64];
                    sum.x += v.x; sum.y += v.y; sum.z += v.z; sum.w += v.w;
                }
            }
            if (what == 1) qs[half * 64 + w * 32 + lane] = sum;
            else {
                const float x[4] = {sum.x, sum.y, sum.z, sum.w};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int r = half * 16 + g8 + (e >> 1) * 8, c = w * 8 + t4 * 2 + (e & 1);
                    split_tf32(val[r * NC + c] - x[e], Uh[r * SROW + c], Ul[r * SROW + c]);
                }
            }
        }
        __syncthreads();                            // U and Q S are there; S has been read
        if (owns) {
            float up[2][3][4] = {};
            product(up, rec_k + warp * (CT >> 3) * 128, Uh, Ul, 0, CT >> 3, lane);
            const float p0 = rec_p[warp * 16 + g8], p1 = rec_p[warp * 16 + g8 + 8];
#pragma unroll
            for (int w = 0; w < 2; ++w)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int r = warp * 16 + g8 + (e >> 1) * 8, c = w * 8 + t4 * 2 + (e & 1);
                    s[w][e] = fmaf(e < 2 ? p0 : p1, s[w][e], up[w][0][e] + (up[w][1][e] + up[w][2][e]));
                    split_tf32(s[w][e], Sh[r * SROW + c], Sl[r * SROW + c]);
                }
        }
        if (warp >= 14) {                           // the chunk's outputs: B U joins Q S
            const int half = warp - 14;
            float acc[2][3][4] = {};
            product(acc, rec_b + half * (CT >> 3) * 128, Uh, Ul, 0, CT >> 3, lane);
            const int t = begin + p * CT;
#pragma unroll
            for (int w = 0; w < 2; ++w) {
                const float4 o = qs[half * 64 + w * 32 + lane], u = chains(acc[w]);
                const float x[4] = {o.x + u.x, o.y + u.y, o.z + u.z, o.w + u.w};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int r = half * 16 + g8 + (e >> 1) * 8, c = j0 + w * 8 + t4 * 2 + (e & 1);
                    if (t + r < t1 && c < dv) out[((size_t)(t + r) * H + h) * dv + c] = x[e];
                }
            }
        }
        __syncthreads();                            // the stage is free
        request(p + STAGES);
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
    for (int w = 0; w < 2; ++w)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int r = warp * 16 + g8 + (e >> 1) * 8, c = w * 8 + t4 * 2 + (e & 1);
            if (owns && j0 + c < dv && r < dk) row[(size_t)(j0 + c) * dk + r] = s[w][e];
        }
}

template <typename K> int reserve(K kernel, size_t bytes, size_t& granted) {
    if (bytes <= 40 * 1024 || bytes <= granted) return 0;
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
    if (e != cudaSuccess) LP_REFUSE("chunked_recurrence: cannot reserve %zu bytes of shared memory: %s", bytes, cudaGetErrorString(e));
    granted = bytes;
    return 0;
}

}  // namespace

extern "C" int lp_chunked_tokens() { return CT; }
// Floats that one chunk of one head needs: a record for the second kernel, and the columns of U.
extern "C" int lp_chunked_record_floats(int dk, int delta) { return record_floats(padded(dk), delta != 0); }
extern "C" int lp_chunked_value_floats(int dv) { return value_floats(dv); }

// The recurrence over a step's tokens of B sequences, from and into `state` (float32 [slots, H, dv, dk]). See Inputs for the
// operands. records: float32 [B, chunks, H, record floats], values: float32 [B, chunks, H, value floats]: room for `chunks`
// chunks of every sequence; a step with longer sequences (max_new: the most new tokens of one) runs in several rounds.
extern "C" int lp_chunked_recurrence(const float* proj, int ld, int q_off, int k_off, int v_off, const float* decay, int decay_form,
                                     const float* key_gain, const float* beta, const float* angles, int rd, int interleaved,
                                     float q_scale, float* state, const int* slots, const int* q_start, float* out, int B, int H,
                                     int dk, int dv, int qk_heads, int max_new, int chunks, float* records, float* values,
                                     cudaStream_t stream) {
    if (B <= 0 || max_new <= 0) return 0;
    if (H <= 0 || H > 65535 || B > 65535 || dk <= 0 || dk > MAX_DK || dv <= 0) LP_REFUSE("chunked_recurrence: %d sequences, %d heads of %d x %d (at most %d key channels)", B, H, dk, dv, MAX_DK);
    if (qk_heads <= 0) qk_heads = H;
    if (H % qk_heads) LP_REFUSE("chunked_recurrence: %d heads over %d query / key heads", H, qk_heads);
    if (q_off < 0 || k_off < 0 || v_off < 0 || q_off + qk_heads * dk > ld || k_off + qk_heads * dk > ld || v_off + H * dv > ld)
        LP_REFUSE("chunked_recurrence: slices at %d, %d, %d do not fit rows of %d", q_off, k_off, v_off, ld);
    if (decay_form < DECAY_CHANNEL || decay_form > DECAY_FIXED) LP_REFUSE("chunked_recurrence: decay form %d", decay_form);
    if (rd < 0 || rd > dk || (rd & 1) || (rd > 0 && !angles)) LP_REFUSE("chunked_recurrence: a rotation over %d of %d channels", rd, dk);
    if (chunks <= 0 || !records || !values) LP_REFUSE("chunked_recurrence: room for %d chunks", chunks);
    if ((((uintptr_t)records | (uintptr_t)values) & 15) != 0) LP_REFUSE("chunked_recurrence: buffers must be aligned to 16 bytes");
    const Inputs in{proj, ld, q_off, k_off, v_off, decay, decay_form, key_gain, beta, (const float2*)angles, rd, interleaved, q_scale,
                    H, dk, dv, H / qk_heads};
    const int dkp = padded(dk), delta = beta ? 1 : 0;
    const size_t smem_p = ((size_t)(3 * CT + 3 * HB) * (dkp + 4) + 2 * CT * CT + CT) * sizeof(float);
    const size_t stage = (size_t)(record_floats(dkp, delta) + CT * NC) * sizeof(float);
    const size_t kept = (size_t)(dkp + CT) * SROW * 2 * sizeof(float) + (16 * 64 + 128) * sizeof(float4);
    const bool two = kept + 2 * stage <= MAX_SMEM;
    const size_t smem_c = kept + (two ? 2 : 1) * stage;
    auto prepare = dk <= 64 ? prepare_kernel<4> : dk <= 128 ? prepare_kernel<8> : prepare_kernel<16>;
    const int size = dk <= 64 ? 0 : dk <= 128 ? 1 : 2;
    auto carry = two ? carry_kernel<2> : carry_kernel<1>;
    static size_t granted_p[3] = {}, granted_c[2] = {};       // what each kernel has been allowed so far
    int rc = reserve(prepare, smem_p, granted_p[size]);
    if (rc) return rc;
    rc = reserve(carry, smem_c, granted_c[two ? 1 : 0]);
    if (rc) return rc;
    const int total = (max_new + CT - 1) / CT;
    for (int first = 0; first < total; first += chunks) {
        const int here = total - first < chunks ? total - first : chunks;
        lp_launch(prepare, dim3(here, H, B), THREADS, smem_p, stream, in, q_start, first, chunks, records, values);
        rc = lp_check_launch("chunked_recurrence (prepare)");
        if (rc) return rc;
        lp_launch(carry, dim3((dv + NC - 1) / NC, H, B), CARRY_THREADS, smem_c, stream, state, slots, q_start, first, chunks,
                  (const float*)records, (const float*)values, out, H, dk, dv, delta);
        rc = lp_check_launch("chunked_recurrence (carry)");
        if (rc) return rc;
    }
    return 0;
}
