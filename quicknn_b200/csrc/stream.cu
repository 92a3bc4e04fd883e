// The float32 residual stream of layers that norm what a sublayer gives, scale it, add it, and may then average over depth.
//
//   qnn_stream_update   X = resid + mult * rmsnorm(y; w_post);  X -> resid_out
//                       with a history:  Z = sum_(j < n) a_j X_j + a_n X,  Z -> avg_out   (X_j: rows that earlier layers left)
//                       out_next = rmsnorm(Z or X; w_next), if asked for
//                       with a filter (decode steps, a row per sequence): h = out_next + conv(out_next), the causal
//                       convolution of short_conv.cu over the sequence's last normed rows, in the place of out_next
//   y may come in `terms` rows per row (the outputs of a row's experts), summed in their order.
//
// One block per row; the row stays in registers between its sums where it fits, eight columns per access where rows allow.
// Earlier layers' rows are read in the order of the layers and each is used once.  All sums are float32.
#include "common.cuh"

using namespace qnn;

namespace {

struct Update {
    const float* resid;
    const void* y;
    const void* w_post;
    const void* w_next;
    float* resid_out;
    const float* hist;        // [n_hist][rows][H]; null: no average
    const void* numbers;      // [n_hist + 1]
    float* avg_out;
    void* out_next;
    const void* conv;         // [H, taps]; null: no convolution
    float* ring;              // slot s: ring + s * slot_stride, [taps][H]: position p in row p mod taps
    const int* tok_pos;
    const int* slots;
    long long hist_stride, slot_stride;
    int terms, conv_dt, taps;
    int y_dt, wp_dt, wn_dt, num_dt, out_dt, n_hist, H;
    float mult, eps_post, off_post, eps_next, off_next;
};

// Eight consecutive values of either element type as they lie in memory: a load that nothing waits for until it is unpacked.
struct Raw8 {
    uint4 a, b;
    __device__ __forceinline__ void load(const void* p, int dt, size_t i) {
        if (dt == QNN_DT_BF16) {
            a = *reinterpret_cast<const uint4*>((const bf16*)p + i);
        } else {
            a = *reinterpret_cast<const uint4*>((const float*)p + i);
            b = *reinterpret_cast<const uint4*>((const float*)p + i + 4);
        }
    }
    __device__ __forceinline__ void unpack(int dt, float* o) const {
        const uint32_t w[8] = {a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w};
#pragma unroll
        for (int e = 0; e < 8; ++e)
            o[e] = dt == QNN_DT_BF16 ? __uint_as_float((e & 1) ? (w[e >> 1] & 0xffff0000u) : (w[e >> 1] << 16)) : __uint_as_float(w[e]);
    }
};

// TAPS > 0: h = n + conv(n), that many taps, of the normed row n (rounded as it is stored), a row per sequence; the row's n joins the ring.
// What waits for no sum (weights before the wait for the kernel in front; the ring's earlier rows; the earlier layers' rows,
// summed in the order of the layers) is asked for before the first sum.
constexpr int MAX_TAPS = 4;
template <int TAPS>
__global__ void __launch_bounds__(TAPS > 0 ? 512 : 1024) stream_update_vec_kernel(const Update u) {
    constexpr bool CONV = TAPS > 0;
    constexpr int CH = 1;             // groups of eight columns per thread
    __shared__ float red[32];
    const size_t base = (size_t)blockIdx.x * u.H;
    const int nchunks = u.H >> 3;
    float v[CH][8], r[CH][8], z[CH][8];
    Raw8 g1[CH], g2[CH], wr[CONV ? TAPS : 1];
    float prev[TAPS > 1 ? TAPS - 1 : 1][8];
    const bool in0 = (int)threadIdx.x < nchunks;
#pragma unroll
    for (int i = 0; i < CH; ++i) {                       // weights are written by no kernel of the step
        const int c = threadIdx.x + i * blockDim.x;
        if (c < nchunks) {
            g1[i].load(u.w_post, u.wp_dt, (size_t)c * 8);
            if (u.out_next != nullptr) g2[i].load(u.w_next, u.wn_dt, (size_t)c * 8);
        }
    }
    int slot = -1, pos = 0;
    float* ring = nullptr;
    if constexpr (CONV) {                                // CH = 1; [channel][tap], taps * 8 numbers in a row
        slot = u.slots[blockIdx.x];
        pos = u.tok_pos[blockIdx.x];
        ring = u.ring + (size_t)(slot < 0 ? 0 : slot) * u.slot_stride + threadIdx.x * 8;
        if (in0)
#pragma unroll
            for (int j = 0; j < TAPS; ++j) wr[j].load(u.conv, u.conv_dt, (size_t)threadIdx.x * 8 * TAPS + j * 8);
    }
    const float a_last = u.hist != nullptr ? load_as_f(u.numbers, u.num_dt, u.n_hist) : 1.f;
    pdl_wait();
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < CH; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
#pragma unroll
        for (int e = 0; e < 8; ++e) v[i][e] = r[i][e] = z[i][e] = 0.f;
        if (c < nchunks) {
            const size_t yat = (size_t)blockIdx.x * u.terms * u.H + (size_t)c * 8, at = base + (size_t)c * 8;
            Raw8 y0, y1;
            y0.load(u.y, u.y_dt, yat);
            if (u.terms > 1) y1.load(u.y, u.y_dt, yat + u.H);
            load8_as_f(u.resid, QNN_DT_F32, at, r[i]);
            y0.unpack(u.y_dt, v[i]);
            for (int k = 1; k < u.terms; ++k) {
                float t[8];
                y1.unpack(u.y_dt, t);
                if (k + 1 < u.terms) y1.load(u.y, u.y_dt, yat + (size_t)(k + 1) * u.H);
#pragma unroll
                for (int e = 0; e < 8; ++e) v[i][e] += t[e];
            }
            if (u.hist != nullptr) {
#pragma unroll 4
                for (int j = 0; j < u.n_hist; ++j) {
                    float h[8];
                    load8_as_f(u.hist, QNN_DT_F32, (size_t)j * u.hist_stride + at, h);
                    const float a = load_as_f(u.numbers, u.num_dt, j);
#pragma unroll
                    for (int e = 0; e < 8; ++e) z[i][e] = fmaf(a, h[e], z[i][e]);
                }
            }
        }
#pragma unroll
        for (int e = 0; e < 8; ++e) ss += v[i][e] * v[i][e];
    }
    if constexpr (CONV) {
#pragma unroll
        for (int d = 1; d < TAPS; ++d) {                 // prev[d - 1]: the row d positions back
            if (in0 && slot >= 0 && pos - d >= 0) load8_as_f(ring + (size_t)((pos - d) % TAPS) * u.H, QNN_DT_F32, 0, prev[d - 1]);
            else
#pragma unroll
                for (int e = 0; e < 8; ++e) prev[d - 1][e] = 0.f;
        }
    }
    ss = block_sum(ss, red);
    const float inv = rsqrtf(ss / (float)u.H + u.eps_post);
    float ss2 = 0.f;
#pragma unroll
    for (int i = 0; i < CH; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c >= nchunks) continue;
        const size_t at = base + (size_t)c * 8;
        float w1[8];
        g1[i].unpack(u.wp_dt, w1);
#pragma unroll
        for (int e = 0; e < 8; ++e) r[i][e] += u.mult * (v[i][e] * inv * (w1[e] + u.off_post));
        store8_from_f(u.resid_out, QNN_DT_F32, at, r[i]);
        if (u.hist != nullptr) {
#pragma unroll
            for (int e = 0; e < 8; ++e) r[i][e] = fmaf(a_last, r[i][e], z[i][e]);
            store8_from_f(u.avg_out, QNN_DT_F32, at, r[i]);
        }
#pragma unroll
        for (int e = 0; e < 8; ++e) ss2 += r[i][e] * r[i][e];
    }
    if (u.out_next == nullptr) return;
    ss2 = block_sum(ss2, red);
    const float inv2 = rsqrtf(ss2 / (float)u.H + u.eps_next);
#pragma unroll
    for (int i = 0; i < CH; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c >= nchunks) continue;
        float o[8], w2[8];
        g2[i].unpack(u.wn_dt, w2);
#pragma unroll
        for (int e = 0; e < 8; ++e) o[e] = r[i][e] * inv2 * (w2[e] + u.off_next);
        if constexpr (CONV) {
            if (slot >= 0) {
                if (u.out_dt == QNN_DT_BF16)
#pragma unroll
                    for (int e = 0; e < 8; ++e) o[e] = __bfloat162float(__float2bfloat16_rn(o[e]));
                store8_from_f(ring + (size_t)(pos % TAPS) * u.H, QNN_DT_F32, 0, o);
                float acc[8], wv[TAPS * 8];
#pragma unroll
                for (int j = 0; j < TAPS; ++j) wr[j].unpack(u.conv_dt, wv + j * 8);
#pragma unroll
                for (int e = 0; e < 8; ++e) acc[e] = 0.f;
#pragma unroll
                for (int d = TAPS - 1; d >= 0; --d)      // the oldest tap first
#pragma unroll
                    for (int e = 0; e < 8; ++e)
                        acc[e] = fmaf(wv[e * TAPS + (TAPS - 1 - d)], d == 0 ? o[e] : prev[d > 0 ? d - 1 : 0][e], acc[e]);
#pragma unroll
                for (int e = 0; e < 8; ++e) o[e] += acc[e];
            }
        }
        store8_from_f(u.out_next, u.out_dt, base + (size_t)c * 8, o);
    }
}

// Any width: a column at a time, each thread re-reads only what it wrote itself.
__global__ void stream_update_kernel(const Update u) {
    __shared__ float red[32];
    pdl_wait();
    const size_t base = (size_t)blockIdx.x * u.H;
    auto y_of = [&](int i) {
        const size_t at = (size_t)blockIdx.x * u.terms * u.H + i;
        float v = load_as_f(u.y, u.y_dt, at);
        for (int k = 1; k < u.terms; ++k) v += load_as_f(u.y, u.y_dt, at + (size_t)k * u.H);
        return v;
    };
    float ss = 0.f;
    for (int i = threadIdx.x; i < u.H; i += blockDim.x) {
        const float v = y_of(i);
        ss += v * v;
    }
    ss = block_sum(ss, red);
    const float inv = rsqrtf(ss / (float)u.H + u.eps_post);
    float ss2 = 0.f;
    for (int i = threadIdx.x; i < u.H; i += blockDim.x) {
        float r = u.resid[base + i] +
                  u.mult * (y_of(i) * inv * (load_as_f(u.w_post, u.wp_dt, i) + u.off_post));
        u.resid_out[base + i] = r;
        if (u.hist != nullptr) {
            float z = 0.f;
            for (int j = 0; j < u.n_hist; ++j)
                z = fmaf(load_as_f(u.numbers, u.num_dt, j), u.hist[(size_t)j * u.hist_stride + base + i], z);
            r = fmaf(load_as_f(u.numbers, u.num_dt, u.n_hist), r, z);
            u.avg_out[base + i] = r;
        }
        ss2 += r * r;
    }
    if (u.out_next == nullptr) return;
    ss2 = block_sum(ss2, red);
    const float inv2 = rsqrtf(ss2 / (float)u.H + u.eps_next);
    const float* from = u.hist != nullptr ? u.avg_out : u.resid_out;
    for (int i = threadIdx.x; i < u.H; i += blockDim.x)
        store_from_f(u.out_next, u.out_dt, base + i, from[base + i] * inv2 * (load_as_f(u.w_next, u.wn_dt, i) + u.off_next));
}

}  // namespace

// resid may be resid_out (in place).  hist (null: no average): rows of n_hist earlier layers, hist_stride floats from one
// layer's rows to the next's; numbers: n_hist + 1 of them, the last one for X; avg_out may be resid but not resid_out.
// w_next / out_next null: no norm follows.  terms: rows of y per row, summed.  conv (null: none; needs out_next, rows of
// whole eights on 16 bytes, at most 4096 columns and four taps, else QNN_ERR_UNSUPPORTED): row t is the next token, at tok_pos[t], of the sequence in slots[t].
QNN_API int qnn_stream_update(const float* resid, const void* y, int y_dt, int terms, float mult, const void* w_post, int wp_dt,
                              float eps_post, int unit_post, float* resid_out, const float* hist, long long hist_stride,
                              int n_hist, const void* numbers, int num_dt, float* avg_out, const void* w_next, int wn_dt,
                              float eps_next, int unit_next, void* out_next, int out_dt, const void* conv, int conv_dt,
                              int taps, float* ring, long long slot_stride, const int* tok_pos, const int* slots, int T, int H,
                              cudaStream_t st) {
    if (T <= 0) return 0;
    if (H <= 0 || terms < 1 || (conv != nullptr && (out_next == nullptr || ring == nullptr || taps < 1 || slot_stride < (long long)taps * H)))
        return QNN_ERR_ARGUMENT;
    if (H <= 0 || (out_next != nullptr && w_next == nullptr)) return QNN_ERR_ARGUMENT;
    if (hist != nullptr && (n_hist < 0 || numbers == nullptr || avg_out == nullptr || avg_out == resid_out)) return QNN_ERR_ARGUMENT;
    Update u;
    u.resid = resid; u.y = y; u.w_post = w_post; u.w_next = w_next; u.resid_out = resid_out; u.hist = hist;
    u.numbers = numbers; u.avg_out = avg_out; u.out_next = out_next; u.hist_stride = hist_stride;
    u.y_dt = y_dt; u.wp_dt = wp_dt; u.wn_dt = wn_dt; u.num_dt = num_dt; u.out_dt = out_dt; u.n_hist = n_hist; u.H = H;
    u.mult = mult; u.eps_post = eps_post; u.off_post = unit_post ? 1.f : 0.f; u.eps_next = eps_next;
    u.off_next = unit_next ? 1.f : 0.f;
    u.terms = terms; u.conv = conv; u.conv_dt = conv_dt; u.taps = taps; u.ring = ring; u.slot_stride = slot_stride;
    u.tok_pos = tok_pos; u.slots = slots;
    const uintptr_t all = (uintptr_t)resid | (uintptr_t)y | (uintptr_t)w_post | (uintptr_t)w_next | (uintptr_t)resid_out |
                          (uintptr_t)hist | (uintptr_t)avg_out | (uintptr_t)out_next | (uintptr_t)ring;
    if ((H & 7) == 0 && (all & 15) == 0 && (hist_stride & 3) == 0 && (slot_stride & 3) == 0 && H <= 8 * 1024) {
        const int threads = ((H >> 3) + 31) / 32 * 32;
        if (conv != nullptr) {
            if (threads > 512 || taps > MAX_TAPS || ((uintptr_t)conv & 15)) return QNN_ERR_UNSUPPORTED;
            if (taps == 4) launch_pdl(stream_update_vec_kernel<4>, dim3(T), dim3(threads), 0, st, u);
            else if (taps == 3) launch_pdl(stream_update_vec_kernel<3>, dim3(T), dim3(threads), 0, st, u);
            else if (taps == 2) launch_pdl(stream_update_vec_kernel<2>, dim3(T), dim3(threads), 0, st, u);
            else launch_pdl(stream_update_vec_kernel<1>, dim3(T), dim3(threads), 0, st, u);
        } else {
            launch_pdl(stream_update_vec_kernel<0>, dim3(T), dim3(threads), 0, st, u);
        }
        QNN_LAUNCH_CHECK();
    }
    if (conv != nullptr) return QNN_ERR_UNSUPPORTED;
    launch_pdl(stream_update_kernel, dim3(T), dim3(H >= 2048 ? 512 : (H >= 512 ? 256 : 128)), 0, st, u);
    QNN_LAUNCH_CHECK();
}
