// Attention with several softmax maps per head over the same values.
//
//   qnn_map_prep         packs the rows of a stacked q | k | v product for the attention kernels, which know one query per head:
//                        query head h, map m becomes query head h * maps + m of `hd` columns with its `dim` numbers at column
//                        m * dim and zeros elsewhere; a key head keeps its maps side by side (maps * dim columns, zeros behind),
//                        so a map's query meets its own map's key and the keys and values of a head are cached once, whatever the
//                        number of maps.  Queries are multiplied by 1 + coef ln(floor((p + 1) / every) + 1) at position p
//                        (coef 0: not).  Keys and values go to the cache line as well.
//   qnn_map_difference   per head: o = a_1 - lambda a_2;  o / sqrt(mean(o^2) + eps) * scale over the head's vdim columns
//
// float32 between load and store.  A block per row packs, a warp per (row, head) subtracts.
#include "common.cuh"

using namespace qnn;

namespace {

// VEC elements at a time: every head size, every pitch in whole VECs
template <typename T, int VEC>
__global__ void map_prep_kernel(const T* __restrict__ src, long long lds, T* __restrict__ dst, long long ldd, int nq, int nk,
                                int maps, int dim, int vdim, int hd, float coef, float every, const int* __restrict__ tok_pos,
                                const int* __restrict__ tok_slot, T* __restrict__ k_pool, T* __restrict__ v_pool,
                                const int* __restrict__ page_table, int max_pages, int page_size, int ring,
                                const int* __restrict__ slot_len, int write_cache, int with_kv) {
    pdl_wait();
    const int t = blockIdx.x, pos = tok_pos[t], slot = tok_slot[t];
    const T* row = src + (size_t)t * lds;
    T* out = dst + (size_t)t * ldd;
    const float temp = coef != 0.f ? 1.f + coef * logf(floorf(__fdiv_rn((float)(pos + 1), every)) + 1.f) : 1.f;
    bool wr = write_cache && slot >= 0;
    if (wr && ring > 0 && pos + ring < slot_len[slot]) wr = false;
    size_t cell = 0;
    if (wr) {
        const int r = ring > 0 ? pos % ring : pos;
        cell = ((size_t)page_table[(size_t)slot * max_pages + r / page_size] * nk * page_size + (r % page_size)) * hd;
    }
    const int per = hd / VEC, nqm = nq * maps;
    const size_t head_stride = (size_t)page_size * hd;
    const int k0 = nq * maps * dim, v0 = k0 + nk * maps * dim;
    // units: query heads, then (key heads, value heads) where somebody wants them
    const int total = (nqm + (with_kv || wr ? 2 * nk : 0)) * per;
    for (int i = threadIdx.x; i < total; i += blockDim.x) {
        const int u = i / per, c = (i - u * per) * VEC;
        int from = -1;                                          // source column, or zeros
        bool query = u < nqm, value = false;
        if (query) {
            const int m = u % maps, d = c - m * dim;
            if (d >= 0 && d < dim) from = u * dim + d;          // head h, map m lies at (h * maps + m) * dim
        } else {
            const int w = u - nqm;
            value = w >= nk;
            const int g = value ? w - nk : w;
            if (c < (value ? vdim : maps * dim)) from = value ? v0 + g * vdim + c : k0 + g * maps * dim + c;
        }
        float v[8];
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[e] = 0.f;
        if (VEC == 8) {
            if (from >= 0) {
                if (sizeof(T) == 2) load8_as_f(row, QNN_DT_BF16, from, v);
                else load8_as_f(row, QNN_DT_F32, from, v);
            }
        } else if (from >= 0) {
            v[0] = to_f(row[from]);
        }
        if (query && coef != 0.f)
#pragma unroll
            for (int e = 0; e < VEC; ++e) v[e] *= temp;
        const int dt = sizeof(T) == 2 ? QNN_DT_BF16 : QNN_DT_F32;
        if (query || with_kv) {
            if (VEC == 8) store8_from_f(out, dt, (size_t)u * hd + c, v);
            else out[(size_t)u * hd + c] = from_f<T>(v[0]);
        }
        if (!query && wr) {
            const int w = u - nqm, g = value ? w - nk : w;
            T* pool = value ? v_pool : k_pool;
            if (VEC == 8) store8_from_f(pool, dt, cell + (size_t)g * head_stride + c, v);
            else pool[cell + (size_t)g * head_stride + c] = from_f<T>(v[0]);
        }
    }
}

template <typename T, bool VEC>
__global__ void map_difference_kernel(const T* __restrict__ a, long long lda, int hd, T* __restrict__ out, long long ldo, int H,
                                      int vdim, float lambda, float eps, float scale, int rows) {
    pdl_wait();
    const long long unit = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31;
    if (unit >= (long long)rows * H) return;
    const size_t t = unit / H;
    const int h = (int)(unit - (long long)t * H);
    const T* a1 = a + t * lda + (size_t)h * 2 * hd;
    const T* a2 = a1 + hd;
    T* o = out + t * ldo + (size_t)h * vdim;
    if (VEC && vdim <= 256) {                                   // a lane holds eight columns
        constexpr int DT = sizeof(T) == 2 ? QNN_DT_BF16 : QNN_DT_F32;
        const int c = lane * 8;
        float x[8], y[8], ss = 0.f;
#pragma unroll
        for (int e = 0; e < 8; ++e) x[e] = y[e] = 0.f;
        if (c < vdim) {
            load8_as_f(a1, DT, c, x);
            load8_as_f(a2, DT, c, y);
        }
#pragma unroll
        for (int e = 0; e < 8; ++e) {
            x[e] = x[e] - lambda * y[e];
            ss += x[e] * x[e];
        }
        ss = warp_sum(ss);
        const float f = rsqrtf(ss / (float)vdim + eps) * scale;
        if (c < vdim) {
#pragma unroll
            for (int e = 0; e < 8; ++e) x[e] *= f;
            store8_from_f(o, DT, c, x);
        }
        return;
    }
    float ss = 0.f;
    for (int c = lane; c < vdim; c += 32) {
        const float x = to_f(a1[c]) - lambda * to_f(a2[c]);
        ss += x * x;
    }
    ss = warp_sum(ss);
    const float f = rsqrtf(ss / (float)vdim + eps) * scale;
    for (int c = lane; c < vdim; c += 32) o[c] = from_f<T>((to_f(a1[c]) - lambda * to_f(a2[c])) * f);
}

template <typename T>
int prep(const void* src, long long lds, void* dst, long long ldd, int rows, int nq, int nk, int maps, int dim, int vdim, int hd,
         float coef, float every, const int* tok_pos, const int* tok_slot, void* k_pool, void* v_pool, const int* page_table,
         int max_pages, int page_size, int ring, const int* slot_len, int write_cache, int with_kv, cudaStream_t st) {
    const bool vec = dim % 8 == 0 && vdim % 8 == 0 && hd % 8 == 0 && (lds * sizeof(T)) % 16 == 0 && (ldd * sizeof(T)) % 16 == 0 &&
                     (((uintptr_t)src | (uintptr_t)dst | (uintptr_t)k_pool | (uintptr_t)v_pool) & 15) == 0;
    const int work = (nq * maps + 2 * nk) * hd / (vec ? 8 : 1);
    const int threads = work >= 512 ? 256 : 128;
#define QNN_MP(V)                                                                                                               \
    launch_pdl(map_prep_kernel<T, V>, dim3(rows), dim3(threads), 0, st, (const T*)src, lds, (T*)dst, ldd, nq, nk, maps, dim, vdim, \
               hd, coef, every, tok_pos, tok_slot, (T*)k_pool, (T*)v_pool, page_table, max_pages, page_size, ring, slot_len,     \
               write_cache, with_kv)
    if (vec) QNN_MP(8);
    else QNN_MP(1);
#undef QNN_MP
    QNN_LAUNCH_CHECK();
}

}  // namespace

// src: [rows, lds]: nq * maps query pieces of dim columns, nk * maps key pieces, nk values of vdim columns.  dst: [rows, ldd]:
// nq * maps heads of hd columns, with with_kv followed by nk key heads and nk value heads.  hd >= maps * dim and >= vdim.  The
// cache arguments are those of qnn_rope_cache_write.
QNN_API int qnn_map_prep(const void* src, int dtype, long long lds, void* dst, long long ldd, int rows, int nq, int nk, int maps,
                         int dim, int vdim, int hd, float coef, float every, const int* tok_pos, const int* tok_slot, void* k_pool,
                         void* v_pool, const int* page_table, int max_pages, int page_size, int ring, const int* slot_len,
                         int write_cache, int with_kv, cudaStream_t st) {
    if (rows <= 0) return 0;
    if (nq <= 0 || nk <= 0 || maps <= 0 || dim <= 0 || vdim <= 0 || hd < maps * dim || hd < vdim || !(every > 0.f) ||
        lds < (long long)(nq + nk) * maps * dim + (long long)nk * vdim ||
        ldd < ((long long)nq * maps + (with_kv ? 2 * nk : 0)) * hd)
        return QNN_ERR_ARGUMENT;
    if (write_cache && (k_pool == nullptr || v_pool == nullptr || page_table == nullptr || slot_len == nullptr || page_size <= 0))
        return QNN_ERR_ARGUMENT;
    if (dtype == QNN_DT_BF16)
        return prep<bf16>(src, lds, dst, ldd, rows, nq, nk, maps, dim, vdim, hd, coef, every, tok_pos, tok_slot, k_pool, v_pool,
                          page_table, max_pages, page_size, ring, slot_len, write_cache, with_kv, st);
    return prep<float>(src, lds, dst, ldd, rows, nq, nk, maps, dim, vdim, hd, coef, every, tok_pos, tok_slot, k_pool, v_pool,
                       page_table, max_pages, page_size, ring, slot_len, write_cache, with_kv, st);
}

// a: [rows, lda]: per head the two maps' outputs, hd columns each (the first vdim count); out: [rows, ldo], vdim columns a head.
QNN_API int qnn_map_difference(const void* a, long long lda, int hd, void* out, long long ldo, int rows, int H, int vdim,
                               float lambda, float eps, float scale, int dtype, cudaStream_t st) {
    if (rows <= 0) return 0;
    if (H <= 0 || vdim <= 0 || hd < vdim || lda < 2LL * H * hd || ldo < (long long)H * vdim) return QNN_ERR_ARGUMENT;
    const size_t es = dtype == QNN_DT_BF16 ? 2 : 4;
    const bool vec = hd % 8 == 0 && vdim % 8 == 0 && (lda * es) % 16 == 0 && (ldo * es) % 16 == 0 &&
                     (((uintptr_t)a | (uintptr_t)out) & 15) == 0;
    const int warps = 4;
    const dim3 grid((unsigned)(((long long)rows * H + warps - 1) / warps));
#define QNN_MD(T, V) \
    launch_pdl(map_difference_kernel<T, V>, grid, dim3(warps * 32), 0, st, (const T*)a, lda, hd, (T*)out, ldo, H, vdim, lambda, eps, scale, rows)
    if (dtype == QNN_DT_BF16) {
        if (vec) QNN_MD(bf16, true);
        else QNN_MD(bf16, false);
    } else {
        if (vec) QNN_MD(float, true);
        else QNN_MD(float, false);
    }
#undef QNN_MD
    QNN_LAUNCH_CHECK();
}
