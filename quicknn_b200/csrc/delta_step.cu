// One token per sequence through the gated delta rule (formulas: delta_rule.cu), everything between the input product and the
// output product in one kernel: the convolutions over the last inputs with silu, the unit vectors, the gates' products, the state's
// step and read-out, the norm of every head and its gate.
//
//   qnn_delta_step
//
// A cluster of `splits` CTAs has one (sequence, value head); a CTA has `cw` of its value columns.  Everything is asked for
// before the wait for the kernel in front but what that kernel writes: the state (the largest part), the ring of the
// convolution's last inputs, filters, the gates' weights.  The CTAs of a cluster exchange their sums of squares for the
// output norm through distributed shared memory.
#include "delta_rule.cuh"

using namespace qnn;

namespace {

constexpr int STEP_THREADS = 256;

struct StepArgs {
    const void* p;              // rows of the input product: q | k | v | gate
    long long ldp;
    const void* x;              // [B, W]: the layer's normed input, for the gates' products
    const void* w_ba;           // [2 H, W]
    int W, w_dt;
    const void* conv;           // [C, taps]
    int c_dt, taps;
    const float* rate;          // exp(A)
    const float* bias;
    const void* norm;           // [vdim]
    int n_dt;
    float eps, q_scale, unit_eps;
    float* state;               // slot s: state + s * slot_stride: [taps][C]; from float s_off on [H][dim][vdim]
    long long slot_stride, s_off;
    const int* tok_pos;
    const int* slots;
    void* out;                  // [B, ldo]: H * vdim columns
    long long ldo;
    int B, H, G, dim, vdim, cw;
};

__device__ __forceinline__ void cluster_arrive() { asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory"); }
__device__ __forceinline__ void cluster_wait() { asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory"); }
__device__ __forceinline__ unsigned cluster_rank() {
    unsigned r;
    asm volatile("mov.u32 %0, %%cluster_ctarank;" : "=r"(r));
    return r;
}

// VEC: the CTA's columns lie in fours on 16 bytes; RPT: state rows per thread
template <typename T, int RPT, bool VEC>
__global__ void __launch_bounds__(STEP_THREADS)
delta_step_kernel(const StepArgs a, int splits) {
    constexpr int V = VEC ? 4 : 1;
    constexpr int CG = 16;                                    // threads side by side over columns: CG * V columns at most
    constexpr int RG = STEP_THREADS / CG;                     // row groups
    __shared__ float sk[DELTA_MAX_DIM], sq[DELTA_MAX_DIM], sv[CG * V], su[CG * V];
    __shared__ float red[8][6];
    __shared__ float part[2][8][CG * V];
    __shared__ float squares[8];                              // by rank of the cluster
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int split = (int)(blockIdx.x % splits), h = (int)(blockIdx.x / splits), b = blockIdx.y;
    const int g = h / (a.H / a.G), D = a.dim, VD = a.vdim;
    const int c0 = split * a.cw, ncol = max(0, min(a.cw, VD - c0));
    const int C = 2 * a.G * D + a.H * VD;
    const int slot = a.slots[b], pos = a.tok_pos[b];
    const int cg = tid % CG, rg = tid / CG;
    if (splits > 1) cluster_arrive();                         // the other CTAs' shared memory is there (waited for below)
    const bool live = slot >= 0;
    float* base = a.state + (size_t)(live ? slot : 0) * a.slot_stride;
    float* S0 = base + a.s_off + (size_t)h * D * VD + c0;
    // Channels of the convolution that this CTA needs: q of its head, k of its head, its value columns, two or three per thread
    // (dim <= 256).  The last three past inputs and their filter columns are asked for together, older ones one by one.
    const int nch = 2 * D + ncol;
    constexpr int PER = (2 * DELTA_MAX_DIM + CG * V + STEP_THREADS - 1) / STEP_THREADS, NEAR = 3;
    float past[PER], last[PER], near_x[PER][NEAR], near_w[PER][NEAR];
    int chan[PER];
    const int newest = pos % a.taps;                          // the ring's row of this token
#pragma unroll
    for (int e = 0; e < PER; ++e) {
        const int i = tid + e * STEP_THREADS;
        last[e] = 0.f;
        chan[e] = -1;
#pragma unroll
        for (int j = 0; j < NEAR; ++j) near_x[e][j] = near_w[e][j] = 0.f;
        if (i < nch) {
            const int ch = i < D ? g * D + i : (i < 2 * D ? a.G * D + g * D + (i - D) : 2 * a.G * D + h * VD + c0 + (i - 2 * D));
            const size_t f = (size_t)ch * a.taps + a.taps - 1;
            chan[e] = ch;
            last[e] = load_as_f(a.conv, a.c_dt, f);
#pragma unroll
            for (int j = 0; j < NEAR; ++j) {                  // j + 1 tokens ago
                const int r = newest - 1 - j;
                if (live && j + 1 < a.taps && pos - 1 - j >= 0) {
                    near_w[e][j] = load_as_f(a.conv, a.c_dt, f - 1 - j);
                    near_x[e][j] = base[(size_t)(r < 0 ? r + a.taps : r) * C + ch];
                }
            }
        }
    }
    // the state: rows rg, rg + RG, ..; columns cg * V ..
    float S[RPT][V];
#pragma unroll
    for (int r = 0; r < RPT; ++r) {
        const int i = rg + r * RG;
#pragma unroll
        for (int c = 0; c < V; ++c) S[r][c] = 0.f;
        if (live && i < D && cg * V < ncol) {
            if (VEC) {
                const float4 s4 = *reinterpret_cast<const float4*>(S0 + (size_t)i * VD + cg * 4);
                S[r][0] = s4.x; S[r][1 % V] = s4.y; S[r][2 % V] = s4.z; S[r][3 % V] = s4.w;
            } else {
                S[r][0] = S0[(size_t)i * VD + cg];
            }
        }
    }
    const float rate = a.rate[h], bias = a.bias[h];
    const float wn = tid < ncol ? load_as_f(a.norm, a.n_dt, c0 + tid) : 0.f;
    // the gates' weights: the first two pieces of eight per thread stay as they come until the input is there
    const size_t wb = (size_t)h * a.W, wa = (size_t)(a.H + h) * a.W;
    const bool early = sizeof(T) == 2 && a.w_dt == QNN_DT_BF16 && a.W % 8 == 0;
    constexpr int EARLY = 2;
    Vec16<bf16> eb[EARLY], ea[EARLY];
#pragma unroll
    for (int u = 0; u < EARLY; ++u) {
        const int i = (tid + u * STEP_THREADS) * 8;
        eb[u].zero();
        ea[u].zero();
        if (early && i < a.W) {
            eb[u].load((const bf16*)a.w_ba + wb + i);
            ea[u].load((const bf16*)a.w_ba + wa + i);
        }
    }
    pdl_wait();
    const T* prow = (const T*)a.p + (size_t)b * a.ldp;
    const T* xrow = (const T*)a.x + (size_t)b * a.W;
    float raw[PER];
#pragma unroll
    for (int e = 0; e < PER; ++e) raw[e] = chan[e] >= 0 ? to_f(prow[chan[e]]) : 0.f;
    const float z = tid < ncol ? to_f(prow[C + h * VD + c0 + tid]) : 0.f;
    // the gates' products
    float db = 0.f, da = 0.f;
    if (early) {
#pragma unroll
        for (int u = 0; u < EARLY; ++u) {
            const int i = (tid + u * STEP_THREADS) * 8;
            if (i < a.W) {
                float xf[8], f[8], e8[8];
                load8_as_f(xrow, QNN_DT_BF16, i, xf);
                eb[u].unpack(f);
                ea[u].unpack(e8);
#pragma unroll
                for (int j = 0; j < 8; ++j) {
                    db += xf[j] * f[j];
                    da += xf[j] * e8[j];
                }
            }
        }
    }
    if (a.W % 8 == 0) {
        for (int i = (tid + (early ? EARLY * STEP_THREADS : 0)) * 8; i < a.W; i += STEP_THREADS * 8) {
            float xf[8], f[8], e8[8];
            load8_as_f(xrow, sizeof(T) == 2 ? QNN_DT_BF16 : QNN_DT_F32, i, xf);
            load8_as_f(a.w_ba, a.w_dt, wb + i, f);
            load8_as_f(a.w_ba, a.w_dt, wa + i, e8);
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                db += xf[j] * f[j];
                da += xf[j] * e8[j];
            }
        }
    } else {
        for (int i = tid; i < a.W; i += STEP_THREADS) {
            const float xf = to_f(xrow[i]);
            db += xf * load_as_f(a.w_ba, a.w_dt, wb + i);
            da += xf * load_as_f(a.w_ba, a.w_dt, wa + i);
        }
    }
    // the past inputs' part of the convolution, oldest first
#pragma unroll
    for (int e = 0; e < PER; ++e) {
        past[e] = 0.f;
        if (chan[e] >= 0 && live)
            for (int j = min(a.taps - 1, pos); j > NEAR; --j) {
                const int r = newest - j;
                past[e] = fmaf(load_as_f(a.conv, a.c_dt, (size_t)chan[e] * a.taps + a.taps - 1 - j),
                               base[(size_t)(r < 0 ? r + a.taps : r) * C + chan[e]], past[e]);
            }
#pragma unroll
        for (int j = NEAR - 1; j >= 0; --j) past[e] = fmaf(near_w[e][j], near_x[e][j], past[e]);
    }
    // convolution, silu (rounded as a prompt's rows are stored), the ring's newest row
    float ssq = 0.f, ssk = 0.f;
#pragma unroll
    for (int e = 0; e < PER; ++e) {
        const int i = tid + e * STEP_THREADS;
        if (chan[e] >= 0) {
            const float y = to_f(from_f<T>(silu(fmaf(last[e], raw[e], past[e]))));
            if (i < D) { sq[i] = y; ssq += y * y; }
            else if (i < 2 * D) { sk[i - D] = y; ssk += y * y; }
            else sv[i - 2 * D] = y;
            // q and k belong to all heads of the group and all CTAs of a cluster: one of them keeps them
            const bool keeper = i >= 2 * D || (split == 0 && h % (a.H / a.G) == 0);
            if (live && keeper) base[(size_t)newest * C + chan[e]] = raw[e];
        }
    }
    {
        const float s0 = warp_sum(ssq), s1 = warp_sum(ssk), s2 = warp_sum(db), s3 = warp_sum(da);
        if (lane == 0) { red[warp][0] = s0; red[warp][1] = s1; red[warp][2] = s2; red[warp][3] = s3; }
    }
    __syncthreads();
    float tq = 0.f, tk = 0.f, tb = 0.f, ta = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) { tq += red[w][0]; tk += red[w][1]; tb += red[w][2]; ta += red[w][3]; }
    const float fq = rsqrtf(tq + a.unit_eps) * a.q_scale, fk = rsqrtf(tk + a.unit_eps);
    const float beta = beta_of(tb), gate = decay_of(ta, rate, bias);
    // S^T k and S^T q: partial sums over a thread's rows, the two row groups of a warp by shuffle, the warps through shared memory
    float mk[V], mq[V], kr[RPT], kq = 0.f;
#pragma unroll
    for (int c = 0; c < V; ++c) mk[c] = mq[c] = 0.f;
#pragma unroll
    for (int r = 0; r < RPT; ++r) {
        const int i = rg + r * RG;
        const float k1 = i < D ? sk[i] * fk : 0.f, q1 = i < D ? sq[i] * fq : 0.f;
        kr[r] = k1;
        if (cg == 0) kq += k1 * q1;
#pragma unroll
        for (int c = 0; c < V; ++c) {
            mk[c] += k1 * S[r][c];
            mq[c] += q1 * S[r][c];
        }
    }
#pragma unroll
    for (int c = 0; c < V; ++c) {
        mk[c] += __shfl_xor_sync(0xffffffffu, mk[c], 16);
        mq[c] += __shfl_xor_sync(0xffffffffu, mq[c], 16);
        if (lane < CG) {
            part[0][warp][cg * V + c] = mk[c];
            part[1][warp][cg * V + c] = mq[c];
        }
    }
    kq += __shfl_xor_sync(0xffffffffu, kq, 16);
    if (lane == 0) red[warp][4] = kq;
    __syncthreads();
    float o = 0.f;
    if (tid < CG * V) {
        float s0 = 0.f, s1 = 0.f, s2 = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) { s0 += part[0][w][tid]; s1 += part[1][w][tid]; s2 += red[w][4]; }
        const float u = tid < ncol ? beta * (sv[tid] - gate * s0) : 0.f;
        su[tid] = u;
        o = tid < ncol ? gate * s1 + s2 * u : 0.f;
    }
    float oo = o * o;                                         // threads of the first CG * V only: at most two warps
    oo = warp_sum(oo);
    if (lane == 0) red[warp][5] = oo;
    __syncthreads();
    float total = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) total += red[w][5];
    if (splits > 1) {
        cluster_wait();
        if (tid < splits) {                                   // this CTA's sum to every rank
            unsigned local = (unsigned)__cvta_generic_to_shared(&squares[cluster_rank()]), remote;
            asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(local), "r"((unsigned)tid));
            asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(remote), "f"(total) : "memory");
        }
        cluster_arrive();
    }
    // meanwhile the new state
#pragma unroll
    for (int r = 0; r < RPT; ++r) {
        const int i = rg + r * RG;
        if (live && i < D && cg * V < ncol) {
            if (VEC) {
                float4 s4;
                s4.x = gate * S[r][0] + kr[r] * su[cg * V];
                s4.y = gate * S[r][1 % V] + kr[r] * su[cg * V + 1 % V];
                s4.z = gate * S[r][2 % V] + kr[r] * su[cg * V + 2 % V];
                s4.w = gate * S[r][3 % V] + kr[r] * su[cg * V + 3 % V];
                *reinterpret_cast<float4*>(S0 + (size_t)i * VD + cg * 4) = s4;
            } else {
                S0[(size_t)i * VD + cg] = gate * S[r][0] + kr[r] * su[cg];
            }
        }
    }
    if (splits > 1) {
        cluster_wait();
        total = 0.f;
        for (int r = 0; r < splits; ++r) total += squares[r];
    }
    if (tid < ncol) {
        const float y = o * rsqrtf(total / (float)VD + a.eps) * wn;
        ((T*)a.out)[(size_t)b * a.ldo + (size_t)h * VD + c0 + tid] = from_f<T>(live ? y * silu(z) : 0.f);
    }
}

template <typename T, int RPT, bool VEC>
int step_as(const StepArgs& a, int splits, cudaStream_t st) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3((unsigned)(a.H * splits), (unsigned)a.B);
    cfg.blockDim = dim3(STEP_THREADS);
    cfg.stream = st;
    cudaLaunchAttribute attr[2];
    int n = 0;
    if (splits > 1) {
        attr[n].id = cudaLaunchAttributeClusterDimension;
        attr[n].val.clusterDim.x = (unsigned)splits;
        attr[n].val.clusterDim.y = 1;
        attr[n].val.clusterDim.z = 1;
        ++n;
    }
    if (pdl_enabled() && (long long)a.H * splits * a.B <= pdl_max_grid()) {
        attr[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attr[n].val.programmaticStreamSerializationAllowed = 1;
        ++n;
    }
    cfg.attrs = attr;
    cfg.numAttrs = n;
    const cudaError_t rc = cudaLaunchKernelEx(&cfg, delta_step_kernel<T, RPT, VEC>, a, splits);
    if (rc != cudaSuccess) return (int)rc;
    QNN_LAUNCH_CHECK();
}

template <typename T, bool VEC>
int step_rows(const StepArgs& a, int splits, cudaStream_t st) {
    const int rpt = (a.dim + 15) / 16;
    if (rpt <= 4) return step_as<T, 4, VEC>(a, splits, st);
    if (rpt <= 8) return step_as<T, 8, VEC>(a, splits, st);
    return step_as<T, 16, VEC>(a, splits, st);
}

}  // namespace

// p: [B, ldp] rows q | k | v | gate of the input product; x: [B, W] the product's input; w_ba: [2 H, W]; conv: [2 G dim + H vdim,
// taps]; state: slot s at state + s * slot_stride: [taps][channels] the ring of last inputs (position p in row p mod taps), from
// float s_off on [H][dim][vdim]; slots negative: a row of no sequence (its output is zero).  out: [B, ldo] of `dtype`.
QNN_API int qnn_delta_step(const void* p, int dtype, long long ldp, const void* x, int W, const void* w_ba, int w_dt,
                           const void* conv, int c_dt, int taps, const float* rate, const float* bias, const void* norm, int n_dt,
                           float eps, float unit_eps, float q_scale, float* state, long long slot_stride, long long s_off, const int* tok_pos,
                           const int* slots, void* out, long long ldo, int B, int H, int G, int dim, int vdim, cudaStream_t st) {
    if (B <= 0) return 0;
    const long long C = 2LL * G * dim + (long long)H * vdim;
    if (H <= 0 || G <= 0 || H % G || dim <= 0 || vdim <= 0 || taps < 1 || W <= 0 || ldp < C + (long long)H * vdim ||
        s_off < taps * C || slot_stride < s_off + (long long)H * dim * vdim || B > 65535 || ldo < (long long)H * vdim)
        return QNN_ERR_ARGUMENT;
    if (dim > DELTA_MAX_DIM) return QNN_ERR_UNSUPPORTED;
    if (W % 8 == 0 && (((uintptr_t)x | (uintptr_t)w_ba) & 15)) return QNN_ERR_ARGUMENT;
    // columns of a CTA: up to 64 in fours, up to 16 one by one; at most eight CTAs share a head
    const bool vec = vdim % 4 == 0 && s_off % 4 == 0 && slot_stride % 4 == 0 && ((uintptr_t)state & 15) == 0;
    const int most = vec ? 64 : 16;
    int splits = 1;
    while (splits < 8 && (long long)splits * most < vdim) splits *= 2;
    int cw = (vdim + splits - 1) / splits;
    if (vec) cw = (cw + 3) / 4 * 4;
    if (cw > most) return QNN_ERR_UNSUPPORTED;
    StepArgs a = {p, ldp, x, w_ba, W, w_dt, conv, c_dt, taps, rate, bias, norm, n_dt, eps, q_scale, unit_eps, state, slot_stride, s_off,
                  tok_pos, slots, out, ldo, B, H, G, dim, vdim, cw};
    if (dtype == QNN_DT_BF16) return vec ? step_rows<bf16, true>(a, splits, st) : step_rows<bf16, false>(a, splits, st);
    return vec ? step_rows<float, true>(a, splits, st) : step_rows<float, false>(a, splits, st);
}
