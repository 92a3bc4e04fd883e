// Rows of latent attention made ready: the latent normed, the shared key part and every query's part rotated, and the key
// row (which is also the value row) appended to the cache.
//
//   qnn_latent_prep   key row  k = [ rot(x_rot, position) | x_c / rms(x_c) * w | 0 ]     (rot_dim, rank, up to `hd` columns)
//                     query h  q = [ rot(q_rot, position) | q_c | . ]                    the first rot_dim columns turn
//
// Column j of the first rot_dim / 2 pairs with j + rot_dim / 2: (u, v) -> (u cos t - v sin t, v cos t + u sin t), t =
// float32(position) * float32(frequency), sincosf.  The latent's norm and the rotation are float32.
//
// q: rows of pitch ldq; q_out: the same rows (in place) or rows of pitch ldo, to which everything is copied.  k_out: columns
// [k_col, k_col + hd) and [k_col + hd, k_col + 2 hd) of the rows q_out get the key row twice (packed q | k | v); negative: not
// written.  The cache line keeps one row per position; a ring keeps the last `ring` positions.  A block per row.
#include "common.cuh"

using namespace qnn;

namespace {

template <typename T, bool VEC>
__global__ void latent_prep_kernel(const T* __restrict__ a, long long lda, int c_col, int r_col, const void* __restrict__ w,
                                   int w_dt, float eps, int rank, int rot, const float* __restrict__ inv_freq,
                                   const T* q, long long ldq, T* q_out, long long ldo, int H, int hd, int k_col,
                                   const int* __restrict__ tok_pos, const int* __restrict__ tok_slot, T* __restrict__ pool,
                                   const int* __restrict__ page_table, int max_pages, int page_size, int ring,
                                   const int* __restrict__ slot_len, int append) {
    extern __shared__ __align__(16) unsigned char smem[];
    __shared__ float red[32];
    T* key = reinterpret_cast<T*>(smem);                              // [hd]
    float2* turn = reinterpret_cast<float2*>(smem + (((size_t)hd * sizeof(T) + 15) & ~(size_t)15));   // [rot / 2] (cos, sin)
    pdl_wait();
    const int t = blockIdx.x, half = rot / 2;
    const int pos = tok_pos[t], slot = tok_slot[t];
    const T* row = a + (size_t)t * lda;
    // what passes unturned from one buffer to the other waits for nothing below
    const T* qr = q + (size_t)t * ldq;
    T* qo = q_out + (size_t)t * ldo;
    const bool in_place = q == q_out;
    if (VEC && !in_place) {
        constexpr int V = Vec16<T>::N;
        const int cc = (hd - rot) / V;
#pragma unroll 4
        for (int i = threadIdx.x; i < H * cc; i += blockDim.x) {
            const int h = i / cc;
            const size_t at = (size_t)h * hd + rot + (i - h * cc) * V;
            Vec16<T> v;
            v.load(qr + at);
            *reinterpret_cast<decltype(v.raw)*>(qo + at) = v.raw;
        }
    }
    float ss = 0.f;
    for (int i = threadIdx.x; i < rank; i += blockDim.x) {
        const float v = to_f(row[c_col + i]);
        ss += v * v;
    }
    for (int j = threadIdx.x; j < half; j += blockDim.x) {
        float s, c;
        sincosf((float)pos * inv_freq[j], &s, &c);
        turn[j] = make_float2(c, s);
    }
    ss = block_sum(ss, red);                                          // also makes `turn` visible
    const float inv = rsqrtf(ss / (float)rank + eps);
    __syncthreads();
    for (int i = threadIdx.x; i < hd; i += blockDim.x) {
        float v = 0.f;
        if (i < rot) {
            const int j = i < half ? i : i - half;
            const float u = to_f(row[r_col + j]), x = to_f(row[r_col + half + j]);
            v = i < half ? u * turn[j].x - x * turn[j].y : x * turn[j].x + u * turn[j].y;
        } else if (i < rot + rank) {
            v = to_f(row[c_col + i - rot]) * inv * load_as_f(w, w_dt, i - rot);
        }
        key[i] = from_f<T>(v);
    }
    // the queries
    if (VEC) {
        constexpr int V = Vec16<T>::N;
        const int rc = half / V;
        for (int i = threadIdx.x; i < H * rc; i += blockDim.x) {
            const int h = i / rc, e = i - h * rc;
            const size_t head = (size_t)h * hd;
            {
                const int j = e * V;
                Vec16<T> uv, xv;
                uv.load(qr + head + j);
                xv.load(qr + head + half + j);
                float u[V], x[V], p[V], s[V];
                uv.unpack(u);
                xv.unpack(x);
#pragma unroll
                for (int k = 0; k < V; ++k) {
                    const float2 cs = turn[j + k];
                    p[k] = u[k] * cs.x - x[k] * cs.y;
                    s[k] = x[k] * cs.x + u[k] * cs.y;
                }
                Vec16<T>::store(qo + head + j, p);
                Vec16<T>::store(qo + head + half + j, s);
            }
        }
    } else {
        for (int i = threadIdx.x; i < H * half; i += blockDim.x) {
            const int h = i / half, j = i - h * half;
            const size_t head = (size_t)h * hd;
            const float u = to_f(qr[head + j]), x = to_f(qr[head + half + j]);
            qo[head + j] = from_f<T>(u * turn[j].x - x * turn[j].y);
            qo[head + half + j] = from_f<T>(x * turn[j].x + u * turn[j].y);
        }
        if (!in_place)
            for (int i = threadIdx.x; i < H * (hd - rot); i += blockDim.x) {
                const int h = i / (hd - rot), d = rot + i - h * (hd - rot);
                qo[(size_t)h * hd + d] = qr[(size_t)h * hd + d];
            }
    }
    __syncthreads();
    // the key row: beside the queries, and to the cache
    bool wr = append && slot >= 0;
    if (wr && ring > 0 && pos + ring < slot_len[slot]) wr = false;    // a prompt longer than the ring keeps its last positions
    T* cell = nullptr;
    if (wr) {
        const int r = ring > 0 ? pos % ring : pos;
        cell = pool + ((size_t)page_table[(size_t)slot * max_pages + r / page_size] * page_size + (r % page_size)) * hd;
    }
    for (int i = threadIdx.x; i < hd; i += blockDim.x) {
        const T v = key[i];
        if (k_col >= 0) {
            qo[k_col + i] = v;
            qo[k_col + hd + i] = v;
        }
        if (wr) cell[i] = v;
    }
}

template <typename T>
int launch(const void* a, long long lda, int c_col, int r_col, const void* w, int w_dt, float eps, int rank, int rot,
           const float* inv_freq, const void* q, long long ldq, void* q_out, long long ldo, int H, int hd, int k_col,
           const int* tok_pos, const int* tok_slot, void* pool, const int* page_table, int max_pages, int page_size, int ring,
           const int* slot_len, int append, int T_rows, cudaStream_t st) {
    constexpr int V = Vec16<T>::N;
    const bool vec = (rot / 2) % V == 0 && (hd - rot) % V == 0 && (ldq * sizeof(T)) % 16 == 0 && (ldo * sizeof(T)) % 16 == 0 &&
                     (((uintptr_t)q | (uintptr_t)q_out) & 15) == 0;
    const size_t smem = (((size_t)hd * sizeof(T) + 15) & ~(size_t)15) + (size_t)(rot / 2) * sizeof(float2);
    if (smem > 48 * 1024) return QNN_ERR_UNSUPPORTED;
    const int work = H * hd / V;
    const int threads = work >= 256 && T_rows <= 1024 ? 256 : 128;      // many rows: more of them on an SM at once
#define QNN_LP(VV)                                                                                                       \
    launch_pdl(latent_prep_kernel<T, VV>, dim3(T_rows), dim3(threads), smem, st, (const T*)a, lda, c_col, r_col, w, w_dt, \
               eps, rank, rot, inv_freq, (const T*)q, ldq, (T*)q_out, ldo, H, hd, k_col, tok_pos, tok_slot, (T*)pool,     \
               page_table, max_pages, page_size, ring, slot_len, append)
    if (vec) QNN_LP(true);
    else QNN_LP(false);
#undef QNN_LP
    QNN_LAUNCH_CHECK();
}

}  // namespace

QNN_API int qnn_latent_prep(const void* a, int dtype, long long lda, int c_col, int r_col, const void* w, int w_dt, float eps,
                            int rank, int rot, const float* inv_freq, const void* q, long long ldq, void* q_out, long long ldo,
                            int H, int hd, int k_col, const int* tok_pos, const int* tok_slot, void* pool,
                            const int* page_table, int max_pages, int page_size, int ring, const int* slot_len, int append,
                            int T, cudaStream_t st) {
    if (T <= 0) return 0;
    if (rank <= 0 || rot < 0 || (rot & 1) || hd < rank + rot || H <= 0 || ldq < (long long)H * hd ||
        ldo < (k_col >= 0 ? k_col + 2LL * hd : (long long)H * hd) || (append && (pool == nullptr || page_size <= 0)))
        return QNN_ERR_ARGUMENT;
    if (dtype == QNN_DT_BF16)
        return launch<bf16>(a, lda, c_col, r_col, w, w_dt, eps, rank, rot, inv_freq, q, ldq, q_out, ldo, H, hd, k_col, tok_pos,
                            tok_slot, pool, page_table, max_pages, page_size, ring, slot_len, append, T, st);
    return launch<float>(a, lda, c_col, r_col, w, w_dt, eps, rank, rot, inv_freq, q, ldq, q_out, ldo, H, hd, k_col, tok_pos,
                         tok_slot, pool, page_table, max_pages, page_size, ring, slot_len, append, T, st);
}
