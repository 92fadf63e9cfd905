// Plain attention of a batch of query tokens over the paged key/value cache.
//
// One block per (query token, query head). Keys are visited in blocks of 128
// aligned to absolute positions; within a block one thread scores one key, the
// running maximum and sum are updated (online softmax, all float32), then each
// thread owns output features and adds the block's weighted values in increasing
// key order. The order of every sum depends only on the query's position and the
// window, never on how tokens were cut into steps or batched.
//
// Counterpart in the reference: src/main/resources/kernels/cuda/attention.cu:10-108
// (one query, scores in shared memory) and the online-softmax variant
// inference/Attention.java:161-207.
#include "common.cuh"

namespace {

constexpr int KB = 128;       // keys per block = threads per block
constexpr int MAX_HD = 256;

template <typename TQ, typename TKV>
__global__ void __launch_bounds__(KB)
attention_plain_kernel(const TQ* __restrict__ q, TQ* __restrict__ out, const TKV* __restrict__ pages,
                       const int* __restrict__ page_table, int pt_stride, const int* __restrict__ seq_ids,
                       const int* __restrict__ positions, int H, int G, int hd, int page_size, float scale,
                       int window, float softcap, const float* __restrict__ sinks, int keep, int chunk,
                       const float* __restrict__ dist_scale, const float* __restrict__ dist_rate,
                       const float* __restrict__ gate, int gate_ld) {
    __shared__ float qs[MAX_HD];
    __shared__ float prob[KB];
    __shared__ long long row_off[KB];
    __shared__ float scratch[32];

    const int t = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
    const int g = h / (H / G);
    const int seq = seq_ids[t];
    const int pos = positions[t];
    int lo = (window > 0 && pos - window + 1 > 0) ? pos - window + 1 : 0;
    if (chunk > 0) lo = max(lo, pos / chunk * chunk);         // keys of the query's own chunk of positions only
    const float ds = dist_scale ? dist_scale[h] : 0.f, dr = dist_scale ? dist_rate[h] : 0.f;
    // a window may keep a sequence's first `keep` tokens visible as well: keys [0, keep_end) besides [lo, pos]
    const int keep_end = keep < lo ? (keep > 0 ? keep : 0) : lo;
    const int c_lo = (lo / KB) * KB;

    const TQ* qr = q + ((long long)t * H + h) * hd;
    for (int i = tid; i < hd; i += KB) qs[i] = lp_to_float(qr[i]);
    __syncthreads();

    float m = -INFINITY, l = 0.f;
    float acc0 = 0.f, acc1 = 0.f;   // features tid and tid + 128
    const int* pt = page_table + (long long)seq * pt_stride;

    for (int c0 = 0;; c0 += KB) {
        if (c0 >= keep_end && c0 < c_lo) c0 = c_lo;      // the blocks between the kept tokens and the window are not seen
        if (c0 > pos) break;
        const int key = c0 + tid;
        const bool valid = key <= pos && (key >= lo || key < keep_end);
        float sc = -INFINITY;
        if (valid) {
            const int page = pt[key / page_size];
            const long long off = (((long long)page * 2 * G + g) * page_size + (key % page_size)) * hd;
            row_off[tid] = off;
            const TKV* kr = pages + off;
            float dot = 0.f;
            for (int i = 0; i < hd; ++i) dot = fmaf(qs[i], lp_to_float(kr[i]), dot);
            sc = dot * scale;
            if (softcap > 0.f) sc = softcap * tanhf(sc / softcap);
            if (dist_scale) sc -= ds * log1pf(dr * (float)(pos - key));
        }
        const float cmax = lp_block_max(sc, scratch);
        const float m_new = fmaxf(m, cmax);
        const float pr = valid ? expf(sc - m_new) : 0.f;
        prob[tid] = pr;
        const float csum = lp_block_sum(pr, scratch);   // also publishes prob[] and row_off[]
        const float alpha = (m == -INFINITY) ? 0.f : expf(m - m_new);
        l = l * alpha + csum;
        acc0 *= alpha;
        acc1 *= alpha;
        const int nk = (pos - c0 + 1 < KB) ? pos - c0 + 1 : KB;
        const int first = c0 < keep_end ? 0 : (lo > c0 ? lo - c0 : 0);
        const long long v_shift = (long long)G * page_size * hd;    // from a K row to its V row
        if (tid < hd) {
            for (int j = first; j < nk; ++j)
                if (prob[j] > 0.f) acc0 = fmaf(prob[j], lp_to_float(pages[row_off[j] + v_shift + tid]), acc0);
        }
        if (tid + KB < hd) {
            for (int j = first; j < nk; ++j)
                if (prob[j] > 0.f) acc1 = fmaf(prob[j], lp_to_float(pages[row_off[j] + v_shift + tid + KB]), acc1);
        }
        m = m_new;
        __syncthreads();
    }
    // a sink: a learned logit per head that takes part in the softmax's denominator only, once
    if (sinks) {
        const float sk = sinks[h];
        const float m_new = fmaxf(m, sk);
        const float alpha = expf(m - m_new);
        l = l * alpha + expf(sk - m_new);
        acc0 *= alpha;
        acc1 *= alpha;
    }
    // a gate per query token and head multiplies the head's finished output
    const float inv = gate ? 1.0f / (l * (1.0f + expf(-gate[(long long)t * gate_ld + h]))) : 1.0f / l;
    TQ* o = out + ((long long)t * H + h) * hd;
    if (tid < hd) o[tid] = lp_from_float<TQ>(acc0 * inv);
    if (tid + KB < hd) o[tid + KB] = lp_from_float<TQ>(acc1 * inv);
}

}  // namespace

// q, out: [T, H, hd]; pages: [num_pages, 2, G, page_size, hd]; page_table: [B, pt_stride];
// seq_ids, positions: [T]. window <= 0: all keys up to the query's position. softcap > 0: a score s becomes
// softcap * tanh(s / softcap) after the scale. sinks (optional): float32 [H], see the kernel. keep > 0 (with a window):
// the sequence's first `keep` tokens stay visible to every later query, at their true positions. chunk > 0: a query at p
// sees keys from p / chunk * chunk on only. dist_scale, dist_rate (optional, float32 [H] each): a key n positions back
// loses dist_scale[h] * ln(1 + dist_rate[h] * n) of its score. gate (optional, float32, rows of gate_ld values): head h's
// output of query token t is multiplied by sigmoid(gate[t, h]).
extern "C" int lp_attention_plain(const void* q, void* out, int q_dtype, const void* pages, int kv_dtype,
                                  const int* page_table, int pt_stride, const int* seq_ids, const int* positions,
                                  int T, int H, int G, int hd, int page_size, float scale, int window,
                                  float softcap, const float* sinks, int keep, int chunk, const float* dist_scale,
                                  const float* dist_rate, const float* gate, int gate_ld, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (gate && gate_ld < H) LP_REFUSE("attention_plain: rows of %d gates for %d heads", gate_ld, H);
    if ((dist_scale == nullptr) != (dist_rate == nullptr)) LP_REFUSE("attention_plain: a distance bias has a scale and a rate per head");
    if (keep > 0 && window > 0 && chunk > 0) LP_REFUSE("attention_plain: kept first tokens (%d) and chunks (%d) exclude each other", keep, chunk);
    if (H <= 0 || G <= 0 || H % G) LP_REFUSE("attention_plain: %d query heads over %d key heads", H, G);
    if (hd <= 0 || hd > MAX_HD) LP_REFUSE("attention_plain: head size %d (supported: 1..%d)", hd, MAX_HD);
    if (page_size <= 0) LP_REFUSE("attention_plain: page size %d", page_size);
    if (H > 65535) LP_REFUSE("attention_plain: %d heads exceed the grid", H);
    dim3 grid(T, H);
#define LP_LAUNCH_ATT(TQ, TKV)                                                                                 \
    attention_plain_kernel<TQ, TKV><<<grid, KB, 0, stream>>>((const TQ*)q, (TQ*)out, (const TKV*)pages,          \
                                                             page_table, pt_stride, seq_ids, positions, H, G,  \
                                                             hd, page_size, scale, window, softcap, sinks, keep, \
                                                             chunk, dist_scale, dist_rate, gate, gate_ld)
    if (q_dtype == LP_F32 && kv_dtype == LP_F32) LP_LAUNCH_ATT(float, float);
    else if (q_dtype == LP_BF16 && kv_dtype == LP_BF16) LP_LAUNCH_ATT(__nv_bfloat16, __nv_bfloat16);
    else if (q_dtype == LP_F32 && kv_dtype == LP_BF16) LP_LAUNCH_ATT(float, __nv_bfloat16);
    else if (q_dtype == LP_BF16 && kv_dtype == LP_F32) LP_LAUNCH_ATT(__nv_bfloat16, float);
    else LP_REFUSE("attention_plain: dtype codes q=%d kv=%d", q_dtype, kv_dtype);
#undef LP_LAUNCH_ATT
    return lp_check_launch("attention_plain");
}
