// One token per sequence through the recurrent block of a real-gated linear recurrence, in one kernel: the convolution over
// the last inputs, the gates' block-diagonal products, the recurrence and the output gate (formulas: short_conv.cu,
// block_linear.cu, linear_recurrence.cu; this kernel's results are those of the three, bfloat16 rounding of u included).
//
//   qnn_recurrent_step    p rows: y columns, then x columns;  out = scale * S * gelu(y + by)
//
// A CTA owns 32 channels of one part for 16 sequences.  The gates of a channel need u of its whole part, so the CTA forms u of
// the part for its rows (a few multiplications per channel, repeated by the CTAs of the same part) straight into shared
// memory as the A operand; the r and i rows of its channels are the B operand, which arrives by cp.async and is asked for
// before the wait for the kernel in front (weights are written by no kernel).  mma.sync m16n8k16, float32 sums.
// The ring of last inputs holds position p in row p mod taps, so the row that a CTA writes for its own channels is none that
// another CTA reads in the same step.
#include "common.cuh"

using namespace qnn;

namespace {

__device__ __forceinline__ void cp_async_16(unsigned dst, const void* src, bool valid) {
    const int bytes = valid ? 16 : 0;       // 0 source bytes: the destination is zero-filled
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(dst), "l"(src), "r"(bytes));
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;\n" ::); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N)); }
__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], unsigned addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma_16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile(
        "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
        : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

constexpr int ROWS = 16, CH = 32, BK = 64, STAGES = 4, THREADS = 256, ROWB = BK * 2;
constexpr int PER = ROWS * CH / THREADS;          // (row, channel) pairs that a thread finishes
constexpr int W_STAGE = 2 * CH * ROWB;            // r rows, then i rows
constexpr int MAX_PART = 1024;
constexpr int MAX_TAPS = 8;

struct Step {
    const bf16* p;              // rows of pitch ldp; y columns from y_col, x columns from x_col
    const void* xb;             // biases and the filter: any element type
    const void* yb;
    const void* conv;           // [C, taps]
    const void* cb;
    const bf16* w;              // [blocks, 2 * part, part]
    const float* rb;
    const float* ib;
    const float* decay;
    bf16* out;                  // rows of pitch ldo
    float* state;               // slot s: state + s * slot_stride: [taps][C], then [C]
    const int* tok_pos;
    const int* slots;
    long long ldp, ldo, slot_stride;
    int v_dt, y_col, x_col, B, C, part, taps;
    float scale;
};

// TAPS > 0: the number of taps, whose filter then stays in registers as bfloat16 pairs are read eight at a time; 0: any number.
template <int TAPS>
__global__ void __launch_bounds__(THREADS) recurrent_step_kernel(const Step s) {
    extern __shared__ __align__(128) unsigned char smem[];
    const int nk = (s.part + BK - 1) / BK, taps = TAPS > 0 ? TAPS : s.taps;
    unsigned char* sA = smem;                                   // [nk] slabs of 16 rows x 128 bytes, chunks XOR-ed with the row
    unsigned char* sW = smem + (size_t)nk * ROWS * ROWB;        // [STAGES]
    float* logits = reinterpret_cast<float*>(sW);               // [ROWS][2 * CH + 1], once the products are done
    __shared__ int slot_s[ROWS], pos_s[ROWS];
    const int b = blockIdx.z, c0 = blockIdx.x * CH, m0 = blockIdx.y * ROWS;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
    const bf16* wb = s.w + (size_t)b * 2 * s.part * s.part;
    const unsigned wbase = (unsigned)__cvta_generic_to_shared(sW), abase = (unsigned)__cvta_generic_to_shared(sA);
    auto load = [&](int kb) {
        if (kb < nk) {
            const unsigned dst = wbase + (kb % STAGES) * W_STAGE;
#pragma unroll
            for (int i = tid; i < 2 * CH * 8; i += THREADS) {
                const int r = i >> 3, c = i & 7, k = kb * BK + c * 8;
                const int ch = c0 + (r & (CH - 1));
                const bool ok = ch < s.part && k < s.part;
                const bf16* src = ok ? wb + (size_t)((r < CH ? 0 : s.part) + ch) * s.part + k : s.w;
                cp_async_16(dst + r * ROWB + ((c ^ (r & 7)) << 4), src, ok);
            }
        }
        cp_async_commit();
    };
#pragma unroll
    for (int i = 0; i < STAGES - 1; ++i) load(i);
    // A thread forms u of eight channels (chunk `uc` of the part) for every `rstep`-th row.  Filter and biases, and the
    // constants of the (row, channel) pairs that it finishes, are written by no kernel: asked for before the wait.
    const int chunks = nk * 8, rstep = max(1, THREADS / chunks);
    const int live = min(ROWS, s.B - m0);
    float wv[TAPS > 0 ? TAPS * 8 : 1], xb[8], cb[8];
    const int uc = tid % chunks, ur = tid / chunks;
    const bool mine = uc * 8 < s.part && ur < rstep;
    if (mine) {
        const int ch = b * s.part + uc * 8;
        load8_as_f(s.xb, s.v_dt, ch, xb);
        load8_as_f(s.cb, s.v_dt, ch, cb);
        if constexpr (TAPS > 0) {
#pragma unroll
            for (int i = 0; i < TAPS; ++i) load8_as_f(s.conv, s.v_dt, (size_t)ch * TAPS + i * 8, wv + i * 8);   // [channel][tap]
        }
    }
    float dec[PER], rb[PER], ib[PER], yb[PER];
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        const int k = c0 + (tid + i * THREADS) % CH;
        if (k < s.part) {
            const int ch = b * s.part + k;
            dec[i] = s.decay[ch];
            rb[i] = s.rb[ch];
            ib[i] = s.ib[ch];
            yb[i] = load_as_f(s.yb, s.v_dt, ch);
        }
    }
    if (tid < ROWS) {                                           // from the host, before the step
        slot_s[tid] = m0 + tid < s.B ? s.slots[m0 + tid] : -1;
        pos_s[tid] = m0 + tid < s.B ? s.tok_pos[m0 + tid] : 0;
    }
    pdl_wait();
    __syncthreads();
    float old[PER], yv[PER];
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        const int r = (tid + i * THREADS) / CH, k = c0 + (tid + i * THREADS) % CH;
        if (k < s.part && slot_s[r] >= 0) {
            const int ch = b * s.part + k;
            old[i] = s.state[(size_t)slot_s[r] * s.slot_stride + (size_t)taps * s.C + ch];
            yv[i] = __bfloat162float(s.p[(size_t)(m0 + r) * s.ldp + s.y_col + ch]);
        }
    }
    // u of the part, as the A operand; this CTA's own channels also leave their new input in the ring
    for (int i = tid; i < ROWS * chunks; i += THREADS) {        // rows of no sequence, columns beyond the part
        const int r = i / chunks, c = i - r * chunks;
        if (slot_s[r] < 0 || c * 8 >= s.part)
            *reinterpret_cast<uint4*>(sA + (size_t)(c >> 3) * ROWS * ROWB + r * ROWB + (((c & 7) ^ (r & 7)) << 4)) = make_uint4(0u, 0u, 0u, 0u);
    }
    if (mine) {                                                 // (a part has at most MAX_PART / 8 = 128 chunks)
        const int c = uc, k = c * 8, ch = b * s.part + k;
        for (int r = ur; r < live; r += rstep) {
            if (slot_s[r] < 0) continue;
            const int pos = pos_s[r];
            float* ring = s.state + (size_t)slot_s[r] * s.slot_stride + ch;
            float v[8], u[8];
            load8_as_f(s.p, QNN_DT_BF16, (size_t)(m0 + r) * s.ldp + s.x_col + ch, v);
            if constexpr (TAPS > 0) {
                float x[TAPS][8];
#pragma unroll
                for (int j = 0; j + 1 < TAPS; ++j) {
                    const int q = pos - TAPS + 1 + j;
                    if (q >= 0) load8_as_f(ring + (size_t)(q % TAPS) * s.C, QNN_DT_F32, 0, x[j]);
                    else
#pragma unroll
                        for (int e = 0; e < 8; ++e) x[j][e] = 0.f;
                }
#pragma unroll
                for (int e = 0; e < 8; ++e) {
                    v[e] += xb[e];
                    x[TAPS - 1][e] = v[e];
                    u[e] = 0.f;
#pragma unroll
                    for (int j = 0; j < TAPS; ++j) u[e] = fmaf(wv[e * TAPS + j], x[j][e], u[e]);
                    u[e] += cb[e];
                }
            } else {
#pragma unroll
                for (int e = 0; e < 8; ++e) {
                    v[e] += xb[e];
                    u[e] = 0.f;
                }
                for (int j = 0; j < taps; ++j) {                // the order of the taps: oldest first
                    const int q = pos - taps + 1 + j;
                    if (q < 0) continue;
                    float x[8];
                    if (q == pos) {
#pragma unroll
                        for (int e = 0; e < 8; ++e) x[e] = v[e];
                    } else {
                        load8_as_f(ring + (size_t)(q % taps) * s.C, QNN_DT_F32, 0, x);
                    }
#pragma unroll
                    for (int e = 0; e < 8; ++e) u[e] = fmaf(load_as_f(s.conv, s.v_dt, (size_t)(ch + e) * taps + j), x[e], u[e]);
                }
#pragma unroll
                for (int e = 0; e < 8; ++e) u[e] += cb[e];
            }
            if (k >= c0 && k < c0 + CH) store8_from_f(ring + (size_t)(pos % taps) * s.C, QNN_DT_F32, 0, v);
            Vec16<bf16>::store(reinterpret_cast<bf16*>(sA + (size_t)(c >> 3) * ROWS * ROWB + r * ROWB + (((c & 7) ^ (r & 7)) << 4)), u);
        }
    }

    float acc[4] = {0.f, 0.f, 0.f, 0.f};                        // 16 rows x the warp's 8 of the 64 gate rows
    for (int kb = 0; kb < nk; ++kb) {
        cp_async_wait<STAGES - 2>();
        __syncthreads();
        load(kb + STAGES - 1);
        const unsigned sa = abase + kb * ROWS * ROWB, sb = wbase + (kb % STAGES) * W_STAGE;
#pragma unroll
        for (int ks = 0; ks < BK / 16; ks += 2) {
            uint32_t a0[4], a1[4], bf[4];
            const int r = lane & 15, rb_ = warp * 8 + (lane & 7), cb_ = ks * 2 + (lane >> 3);
            ldmatrix_x4(a0, sa + r * ROWB + (((ks * 2 + (lane >> 4)) ^ (r & 7)) << 4));
            ldmatrix_x4(a1, sa + r * ROWB + (((ks * 2 + 2 + (lane >> 4)) ^ (r & 7)) << 4));
            ldmatrix_x4(bf, sb + rb_ * ROWB + ((cb_ ^ (rb_ & 7)) << 4));        // 32 inner elements of the warp's 8 rows
            mma_16816(acc, a0, bf[0], bf[1]);
            mma_16816(acc, a1, bf[2], bf[3]);
        }
    }
    cp_async_wait<0>();
    __syncthreads();
    constexpr int LD = 2 * CH + 1;
#pragma unroll
    for (int e = 0; e < 4; ++e) logits[(g + (e >> 1) * 8) * LD + warp * 8 + t4 * 2 + (e & 1)] = acc[e];
    __syncthreads();
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        const int r = (tid + i * THREADS) / CH, n = (tid + i * THREADS) % CH, k = c0 + n;
        if (r >= live || k >= s.part) continue;
        const int ch = b * s.part + k;
        bf16* dst = s.out + (size_t)(m0 + r) * s.ldo + ch;
        if (slot_s[r] < 0) {
            *dst = __float2bfloat16_rn(0.f);
            continue;
        }
        const float u = __bfloat162float(*reinterpret_cast<const bf16*>(
            sA + (size_t)(k >> 6) * ROWS * ROWB + r * ROWB + ((((k >> 3) & 7) ^ (r & 7)) << 4) + (k & 7) * 2));
        const float la = -dec[i] * (1.f / (1.f + expf(-(logits[r * LD + n] + rb[i]))));
        const float gi = 1.f / (1.f + expf(-(logits[r * LD + CH + n] + ib[i])));
        const float S = fmaf(expf(la), old[i], sqrtf(-expm1f(2.f * la)) * gi * u);
        s.state[(size_t)slot_s[r] * s.slot_stride + (size_t)taps * s.C + ch] = S;
        *dst = __float2bfloat16_rn(s.scale * S * gelu_tanh(yv[i] + yb[i]));
    }
}

}  // namespace

// p, out, w: bfloat16.  v_dt: the element type of the biases xb, yb, cb and the filter.  Row t of p is the next token, at
// position tok_pos[t], of the sequence in slot slots[t] (negative: no sequence, zeros out).  state: [taps * C] numbers of the
// ring, then [C] of the recurrence, per slot.
QNN_API int qnn_recurrent_step(const void* p, long long ldp, int y_col, int x_col, const void* xb, const void* yb, const void* conv,
                               const void* cb, int v_dt, const void* w, const float* rb, const float* ib, const float* decay,
                               float scale, void* out, long long ldo, float* state, long long slot_stride, const int* tok_pos,
                               const int* slots, int B, int C, int part, int taps, cudaStream_t st) {
    if (B <= 0) return 0;
    if (C <= 0 || part <= 0 || C % part || taps < 1 || slot_stride < (long long)(taps + 1) * C || y_col < 0 || x_col < 0 ||
        ldp < (long long)(y_col > x_col ? y_col : x_col) + C || ldo < C)
        return QNN_ERR_ARGUMENT;
    if (part % 8 || part > MAX_PART || taps > MAX_TAPS || x_col % 8 || ldp % 8 || slot_stride % 4 || C % 8 || C / part > 65535 ||
        (B + ROWS - 1) / ROWS > 65535 ||
        (((uintptr_t)p | (uintptr_t)w | (uintptr_t)xb | (uintptr_t)cb | (uintptr_t)state) & 15))
        return QNN_ERR_UNSUPPORTED;
    Step s;
    s.p = (const bf16*)p; s.xb = xb; s.yb = yb; s.conv = conv; s.cb = cb; s.w = (const bf16*)w; s.rb = rb; s.ib = ib;
    s.decay = decay; s.out = (bf16*)out; s.state = state; s.tok_pos = tok_pos; s.slots = slots; s.ldp = ldp; s.ldo = ldo;
    s.slot_stride = slot_stride; s.v_dt = v_dt; s.y_col = y_col; s.x_col = x_col; s.B = B; s.C = C; s.part = part;
    s.taps = taps; s.scale = scale;
    const size_t smem = (size_t)((part + BK - 1) / BK) * ROWS * ROWB + (size_t)STAGES * W_STAGE;
    const dim3 grid((part + CH - 1) / CH, (B + ROWS - 1) / ROWS, C / part);
    static bool configured = false;
    if (!configured) {
        const int most = (MAX_PART / BK) * ROWS * ROWB + STAGES * W_STAGE;
        cudaError_t e = cudaFuncSetAttribute(recurrent_step_kernel<4>, cudaFuncAttributeMaxDynamicSharedMemorySize, most);
        if (e == cudaSuccess) e = cudaFuncSetAttribute(recurrent_step_kernel<0>, cudaFuncAttributeMaxDynamicSharedMemorySize, most);
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    if (taps == 4 && ((uintptr_t)conv & 15) == 0) launch_pdl(recurrent_step_kernel<4>, grid, dim3(THREADS), smem, st, s);
    else launch_pdl(recurrent_step_kernel<0>, grid, dim3(THREADS), smem, st, s);
    QNN_LAUNCH_CHECK();
}
