// Attention over a cached latent: per token the cache keeps one row [c | k_r] (a normed latent of
// `rank` numbers and one rotated key part of `rot` numbers shared by all heads) instead of keys and
// values per head.  The per-head products are moved to the query side: with q_h = [q_plain | q_rot],
//
//   score_h(j) = (q_plain . (W_uk,h c_j) + q_rot . k_r,j) scale = ((W_uk,h^T q_plain) . c_j + q_rot . k_r,j) scale
//   out_h      = W_uv,h (sum_j p_h(j) c_j),   p_h(j) = exp(s_j) / (exp(sink_h) + sum_j' exp(s_j'))
//
// so a query row is [W_uk,h^T q_plain | q_rot] (rank + rot numbers per head, made by a grouped product
// and cw_latent_prepare), all heads read the same cached rows, and the kernel returns sum_j p c_j per
// head for another grouped product to map to the head's value size.  The sink is a learned number per
// head that takes part in the softmax denominator only (no key, no value, not scaled, counted once; a layer may have none).
//
//   cw_latent_prepare    RMS norm of the latent (float32) and rotation of the shared key part (rotation.cuh), written to
//                        the cache row of the token's slot; rotation of the queries' rotated parts
//   cw_latent_attention  causal attention of a flat batch (prompt portions beside single tokens) over the
//                        paged rows; float32 scores, weights and accumulation in both run precisions
#include "request_tiles.cuh"
#include "rotation.cuh"

// down [N, rank + rot] (row stride ldd, float32: the projection's output); q [N, H*(dim + rot)] (row stride ldq, QT: float32
// when one product made both, else T): per head [plain | rotated].  Written: the cache row [normed latent | rotated shared key
// part] of the token's slot, the queries' rotated parts into qa [N, H*(rank+rot)] at [.., rank:] of every head and, with
// q_plain [N, H*dim], their plain parts.
template <typename T, typename QT>
__global__ void __launch_bounds__(256)
latent_prepare_kernel(const float* __restrict__ down, int ldd, const QT* __restrict__ q, int ldq, T* __restrict__ q_plain,
                      T* __restrict__ qa, T* __restrict__ cache, const float* __restrict__ norm_w, Rotation rot,
                      const int* __restrict__ positions, const int* __restrict__ slots, int H, int dim, int rank, int num_slots,
                      float eps, int write_cache, int vec, int* status) {
    extern __shared__ float lp_table[];  // cosines, then sines, of the token's pairs
    __shared__ float scratch[33];
    pdl_wait();
    const int row = blockIdx.x, tid = threadIdx.x;
    const int D = rank + rot.dims, half = rot.dims >> 1;
    float *cs = lp_table, *sn = lp_table + half;
    rotation_table(rot, positions[row], cs, sn);
    const float* dr = down + (size_t)row * ldd;
    int slot = write_cache ? slots[row] : -1;
    if (slot >= num_slots) {
        if (tid == 0) cw_report(status, CW_ST_SLOT_RANGE, row, slot);
        slot = -1;
    }
    float ss = 0.f;
    for (int i = tid; i < rank; i += blockDim.x) ss = fmaf(dr[i], dr[i], ss);
    ss = block_sum(ss, scratch);
    __syncthreads();  // the table is written
    const float inv = 1.0f / sqrtf(ss / (float)rank + eps);
    if (slot >= 0) {
        T* cr = cache + (size_t)slot * D;
        for (int i = tid; i < rank; i += blockDim.x) cr[i] = from_f<T>(dr[i] * inv * norm_w[i]);
        for (int i = tid; i < half; i += blockDim.x) {
            const int a = rank + rotation_first(rot, i), b = rank + rotation_second(rot, i);
            const float u = dr[a], v = dr[b];
            cr[a] = from_f<T>(u * cs[i] - v * sn[i]);
            cr[b] = from_f<T>(v * cs[i] + u * sn[i]);
        }
    }
    const QT* qr = q + (size_t)row * ldq;
    for (int idx = tid; idx < H * half; idx += blockDim.x) {
        const int h = idx / half, i = idx - h * half;
        const int a = rotation_first(rot, i), b = rotation_second(rot, i);
        const QT* from = qr + (size_t)h * (dim + rot.dims) + dim;
        const float u = to_f(from[a]), v = to_f(from[b]);
        T* o = qa + (size_t)row * H * D + (size_t)h * D + rank;
        o[a] = from_f<T>(u * cs[i] - v * sn[i]);
        o[b] = from_f<T>(v * cs[i] + u * sn[i]);
    }
    if (q_plain == nullptr) return;
    T* qp = q_plain + (size_t)row * H * dim;
    if (vec) {  // four entries at a time
        const int quads = dim >> 2;
        for (int idx = tid; idx < H * quads; idx += blockDim.x) {
            const int h = idx / quads, i = (idx - h * quads) * 4;
            Vec4<T>::store(qp + (size_t)h * dim + i, Vec4<QT>::load(qr + (size_t)h * (dim + rot.dims) + i));
        }
        return;
    }
    for (int idx = tid; idx < H * dim; idx += blockDim.x) {
        const int h = idx / dim, i = idx - h * dim;
        qp[idx] = from_f<T>(to_f(qr[(size_t)h * (dim + rot.dims) + i]));
    }
}

extern "C" int cw_latent_prepare(const float* down, int ldd, const void* q, int ldq, int q_float32, void* q_plain, void* qa, void* cache,
                                 const float* norm_w, const float* inv_freq, int interleaved, float amplitude, const int* positions,
                                 const int* slots, int N, int H, int dim, int rot_dims, int rank, int num_slots, float eps,
                                 int write_cache, int dtype, int* status, cudaStream_t stream) {
    if (N == 0) return CW_OK;
    const Rotation rot = {inv_freq, rot_dims, interleaved, amplitude};
    if (N < 0 || H <= 0 || dim < 0 || !rotation_ok(rot, rot_dims) || rank <= 0 || ldd < rank + rot_dims || ldq < H * (dim + rot_dims))
        return CW_ERR_BAD_SIZE;
    if (rot_dims > 8192) return CW_ERR_UNSUPPORTED;
    if (dtype != 0 && dtype != 1) return CW_ERR_BAD_DTYPE;
    const bool wide_q = q_float32 || dtype == 0;  // q's entries are float32
    const int vec = dim % 4 == 0 && rot_dims % 4 == 0 && ldq % 4 == 0 && ((uintptr_t)q & 15) == 0 && ((uintptr_t)q_plain & 15) == 0;
    const dim3 grid(N), block(H * (dim + rot_dims) > 1024 ? 256 : 128);
    const size_t smem = sizeof(float) * (size_t)rot_dims;
    if (dtype == 0)
        return cw_launch_ordered(latent_prepare_kernel<float, float>, grid, block, smem, stream, down, ldd, (const float*)q, ldq, (float*)q_plain,
                                 (float*)qa, (float*)cache, norm_w, rot, positions, slots, H, dim, rank, num_slots, eps, write_cache, vec, status);
    if (wide_q)
        return cw_launch_ordered(latent_prepare_kernel<bf16, float>, grid, block, smem, stream, down, ldd, (const float*)q, ldq, (bf16*)q_plain,
                                 (bf16*)qa, (bf16*)cache, norm_w, rot, positions, slots, H, dim, rank, num_slots, eps, write_cache, vec, status);
    return cw_launch_ordered(latent_prepare_kernel<bf16, bf16>, grid, block, smem, stream, down, ldd, (const bf16*)q, ldq, (bf16*)q_plain,
                             (bf16*)qa, (bf16*)cache, norm_w, rot, positions, slots, H, dim, rank, num_slots, eps, write_cache, vec, status);
}

// One block per (token, group of LA_HB heads).  Keys in chunks of 128, a thread per key for the scores
// (all LA_HB heads at once, so a cached row is read once per group), then a thread per latent column for
// the weighted sum.  The chunking depends on the token's position only, never on the rest of the batch.
#define LA_CH 128
#define LA_HB 4
#define LA_NC 8  // latent columns per thread: rank <= LA_CH * LA_NC
#define LT_MAX_PARTS 128  // runs that the tensor-core form may cut a row's keys in

// max or sum of LA_HB values per thread over the block, in a fixed order
template <bool MAX>
__device__ __forceinline__ void block_reduce_heads(float (&v)[LA_HB], float (*buf)[LA_HB]) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
#pragma unroll
    for (int h = 0; h < LA_HB; ++h) v[h] = MAX ? warp_max(v[h]) : warp_sum(v[h]);
    __syncthreads();
    if (lane == 0)
        for (int h = 0; h < LA_HB; ++h) buf[warp][h] = v[h];
    __syncthreads();
#pragma unroll
    for (int h = 0; h < LA_HB; ++h) {
        float r = buf[0][h];
        for (int w = 1; w < LA_CH / 32; ++w) r = MAX ? fmaxf(r, buf[w][h]) : r + buf[w][h];
        v[h] = r;
    }
}

template <typename T, typename TO>
__global__ void __launch_bounds__(LA_CH)
latent_attention_kernel(const T* __restrict__ qa, TO* __restrict__ out, const T* __restrict__ cache,
                        const int* __restrict__ block_tables, const int* __restrict__ tok_seq,
                        const int* __restrict__ positions, const float* __restrict__ sink, int H, int rank, int rot,
                        int page_size, int max_blocks, int num_pages, float scale, int* status) {
    extern __shared__ float q_s[];  // [LA_HB][D]
    __shared__ float p_s[LA_HB][LA_CH];
    __shared__ int slot_s[LA_CH];
    __shared__ float red_s[LA_CH / 32][LA_HB];
    pdl_wait();
    const int t = blockIdx.x, h0 = blockIdx.y * LA_HB, tid = threadIdx.x;
    const int D = rank + rot;
    const int seq = tok_seq[t];
    const int heads = min(LA_HB, H - h0);
    if (seq < 0) {  // padding row of a fixed-shape batch
        for (int i = tid; i < heads * rank; i += LA_CH) out[((size_t)t * H + h0) * rank + i] = from_f<TO>(0.f);
        return;
    }
    for (int i = tid; i < LA_HB * D; i += LA_CH) {
        const int hb = i / D, d = i % D;
        q_s[i] = hb < heads ? to_f(qa[((size_t)t * H + h0 + hb) * D + d]) : 0.f;
    }
    __syncthreads();
    const int kv_end = positions[t] + 1;
    const int* table = block_tables + (size_t)seq * max_blocks;
    float m[LA_HB], l[LA_HB], acc[LA_HB][LA_NC];
#pragma unroll
    for (int hb = 0; hb < LA_HB; ++hb) {
        m[hb] = -INFINITY;
        l[hb] = 0.f;
#pragma unroll
        for (int c = 0; c < LA_NC; ++c) acc[hb][c] = 0.f;
    }
    for (int c0 = 0; c0 < kv_end; c0 += LA_CH) {
        const int j = c0 + tid;
        float s[LA_HB];
#pragma unroll
        for (int hb = 0; hb < LA_HB; ++hb) s[hb] = -INFINITY;
        int slot = -1;
        if (j < kv_end) {
            const int blk = j / page_size;
            const int page = blk < max_blocks ? table[blk] : -1;
            if (page < 0 || page >= num_pages) {
                cw_report(status, CW_ST_PAGE_RANGE, t, page);
            } else {
                slot = page * page_size + j % page_size;
                const T* kp = cache + (size_t)slot * D;
                float dot[LA_HB] = {};
                for (int d = 0; d < D; ++d) {
                    const float kd = to_f(kp[d]);
#pragma unroll
                    for (int hb = 0; hb < LA_HB; ++hb) dot[hb] = fmaf(q_s[hb * D + d], kd, dot[hb]);
                }
#pragma unroll
                for (int hb = 0; hb < LA_HB; ++hb) s[hb] = dot[hb] * scale;
            }
        }
        slot_s[tid] = slot;
        float top[LA_HB];
#pragma unroll
        for (int hb = 0; hb < LA_HB; ++hb) top[hb] = s[hb];
        block_reduce_heads<true>(top, red_s);
        float p[LA_HB], alpha[LA_HB];
#pragma unroll
        for (int hb = 0; hb < LA_HB; ++hb) {
            const float m_new = fmaxf(m[hb], top[hb]);
            p[hb] = slot >= 0 ? expf(s[hb] - m_new) : 0.f;
            p_s[hb][tid] = p[hb];
            alpha[hb] = m[hb] == -INFINITY ? 0.f : expf(m[hb] - m_new);
            m[hb] = m_new;
        }
        block_reduce_heads<false>(p, red_s);  // (its barriers also order p_s and slot_s before the reads below)
#pragma unroll
        for (int hb = 0; hb < LA_HB; ++hb) {
            l[hb] = l[hb] * alpha[hb] + p[hb];
#pragma unroll
            for (int c = 0; c < LA_NC; ++c) acc[hb][c] *= alpha[hb];
        }
        const int n = min(LA_CH, kv_end - c0);
        for (int jj = 0; jj < n; ++jj) {
            const int sl = slot_s[jj];
            if (sl < 0) continue;
            const T* cp = cache + (size_t)sl * D;
#pragma unroll
            for (int c = 0; c < LA_NC; ++c) {
                const int col = tid + c * LA_CH;
                if (col < rank) {
                    const float cv = to_f(cp[col]);
#pragma unroll
                    for (int hb = 0; hb < LA_HB; ++hb) acc[hb][c] = fmaf(p_s[hb][jj], cv, acc[hb][c]);
                }
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int hb = 0; hb < LA_HB; ++hb) {
        if (hb >= heads) continue;
        const float sk = sink != nullptr ? sink[h0 + hb] : -INFINITY;
        const float top = fmaxf(m[hb], sk);
        const float keep = m[hb] == -INFINITY ? 0.f : expf(m[hb] - top);
        const float denom = l[hb] * keep + (sk == -INFINITY ? 0.f : expf(sk - top));
        const float inv = denom > 0.f ? keep / denom : 0.f;
#pragma unroll
        for (int c = 0; c < LA_NC; ++c) {
            const int col = tid + c * LA_CH;
            if (col < rank) out[((size_t)t * H + h0 + hb) * rank + col] = from_f<TO>(acc[hb][c] * inv);
        }
    }
}

// ---- the same on the tensor cores (bfloat16 cache and queries) -------------------------------------------
// A request's (token, head) pairs are the rows of qa in memory, so a block takes 16 MT consecutive rows of one request,
// whatever the number of heads: the cached rows of its keys are read once for all of them.  MT = 4 (prompt portions): 64 rows,
// four tokens of 16 heads; MT = 1 (single tokens): 16 rows.  Blocks are mapped to (request, rows) by a scan of q_start, so a
// captured step needs nothing from the host; blocks of the latest rows, which see the most keys, come first.  Keys come in
// tiles of KT (cp.async through the block table, two stages).  Eight warps: for the scores MT groups of 16 rows by 8 / MT
// groups of KT MT / 8 keys over the whole row width (mma.sync m16n8k16); maxima and sums meet in shared memory (added in
// warp order); the weights go to shared memory as two bfloat16 halves (p = hi + lo, so the product with the latents carries
// float32 weights to 16 bits of mantissa); for the second product 2 x 4 (MT = 4) or 1 x 8 warps share rows and the
// latent's columns, the cached tile itself being the second operand (read transposed by ldmatrix).
// A row's keys may be cut in `parts` runs of whole tiles (few rows, long contexts): every part then leaves its sums, its
// running maxima and denominators, which latent_merge_kernel adds up.
__device__ __forceinline__ void lt_cp16(void* smem, const void* gmem, bool valid) {
    const unsigned dst = (unsigned)__cvta_generic_to_shared(smem);
    const int bytes = valid ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(gmem), "r"(bytes) : "memory");
}
__device__ __forceinline__ void lt_ldm(unsigned (&r)[4], const void* smem) {
    const unsigned a = (unsigned)__cvta_generic_to_shared(smem);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a) : "memory");
}
__device__ __forceinline__ void lt_ldm2(unsigned (&r)[2], const void* smem) {
    const unsigned a = (unsigned)__cvta_generic_to_shared(smem);
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(a) : "memory");
}
__device__ __forceinline__ void lt_ldm_t(unsigned (&r)[4], const void* smem) {
    const unsigned a = (unsigned)__cvta_generic_to_shared(smem);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a) : "memory");
}
__device__ __forceinline__ void lt_mma(float (&c)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ unsigned lt_pack(bf16 a, bf16 b) {
    return (unsigned)__bfloat16_as_ushort(a) | ((unsigned)__bfloat16_as_ushort(b) << 16);
}

struct LatentArgs {
    const bf16* qa;           // [N*H, D]
    bf16* out;                // [N*H, rank]
    const bf16* cache;        // [slots, D]
    const int* block_tables;  // [S, max_blocks]
    const int* tok_seq;       // [N], < 0: padding
    const int* positions;     // [N]
    const int* q_start;       // [S + 1]
    const float* sink;        // [H] or null
    int N, S, H, rank, rot, page_size, max_blocks, num_pages;
    float scale;
    int parts;
    float* partial;           // parts > 1: [parts, N*H, rank] sums, then [parts, N*H, 2] running maxima and denominators
    int* status;
};

template <int MT>
struct LatentTile {
    static constexpr int ROWS = 16 * MT;
    static constexpr int KT = MT == 1 ? 64 : 48;         // keys per tile
    static constexpr int KW = 8 / MT;                    // groups of keys in the score product
    static constexpr int NS = KT / KW / 8;               // n-tiles of 8 keys per warp there
    static constexpr int RW = MT == 1 ? 1 : 2;           // groups of rows in the second product
    static constexpr int CW = 8 / RW;                    // groups of columns there
    static constexpr int MP = MT / RW;                   // m-tiles per warp there
    static constexpr int NP = 64 / CW;                   // n-tiles of 8 latent columns per warp there: rank <= 8 * 64
    static constexpr int PLD = KT + 8;                   // row of the weights in shared memory, in elements
    static size_t smem(int D) {
        return sizeof(bf16) * ((size_t)(2 * KT + ROWS) * (D + 8) + 2 * (size_t)ROWS * PLD) + sizeof(float) * ROWS * (2 * KW + 2) +
               sizeof(int) * 2 * KT;
    }
};

template <int MT>
__global__ void __launch_bounds__(256, 1)
latent_attention_mma_kernel(const LatentArgs a) {
    using L = LatentTile<MT>;
    constexpr int ROWS = L::ROWS, KT = L::KT, KW = L::KW, NS = L::NS, PLD = L::PLD;
    extern __shared__ __align__(16) unsigned char lt_smem[];
    __shared__ int tile_seq, tile_row0, tile_rows;
    const int H = a.H, rank = a.rank, D = rank + a.rot, LDK = D + 8;
    bf16* Ks = (bf16*)lt_smem;                            // [2][KT][LDK]
    bf16* Qs = Ks + (size_t)2 * KT * LDK;                 // [ROWS][LDK]
    bf16* Phi = Qs + (size_t)ROWS * LDK;                  // [ROWS][PLD]
    bf16* Plo = Phi + ROWS * PLD;
    float* row_max = (float*)(Plo + ROWS * PLD);          // [KW][ROWS]
    float* row_sum = row_max + KW * ROWS;                 // [KW][ROWS]
    float* alpha_s = row_sum + KW * ROWS;                 // [ROWS] what the sums so far are multiplied by when the maximum moves
    float* inv_s = alpha_s + ROWS;                        // [ROWS] what they are multiplied by at the end
    int* slot_s = (int*)(inv_s + ROWS);                   // [2][KT]
    pdl_wait();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, part = blockIdx.y;
    const long long total_rows = (long long)a.N * H;
    if (part == 0) {  // rows of no request (padding of a fixed-shape step) come out as zeros
        const long long first = (long long)blockIdx.x * ROWS, last = min(total_rows, first + ROWS);
        for (long long t = first / H; t * H < last; ++t)
            if (a.tok_seq[t] < 0)
                for (long long i = max(first, t * H) * rank + tid; i < min(last, (t + 1) * H) * rank; i += 256) a.out[i] = __float2bfloat16_rn(0.f);
    }
    if (warp == 0) {  // which request and which of its rows
        const RowTile tile = find_row_tile(blockIdx.x, true, a.q_start, a.tok_seq, a.S, H, ROWS);
        if (lane == 0) {
            tile_seq = tile.seq;
            tile_row0 = tile.row0;
            tile_rows = tile.rows;
        }
    }
    __syncthreads();
    const int seq = tile_seq, row0 = tile_row0, rows = tile_rows;
    if (seq < 0) return;
    const int tok0 = row0 / H, head0 = row0 - tok0 * H, p0 = a.positions[tok0];  // the first row's token, head and position
    const int kv_end = p0 + (head0 + rows - 1) / H + 1;                           // keys that the last row sees
    const int all_tiles = (kv_end + KT - 1) / KT, part_tiles = (all_tiles + a.parts - 1) / a.parts;
    const int t_lo = part * part_tiles, t_hi = min(all_tiles, t_lo + part_tiles);
    float* sums = a.partial + ((size_t)part * total_rows + row0) * rank;
    float* stats = a.partial + (size_t)a.parts * total_rows * rank + ((size_t)part * total_rows + row0) * 2;
    if (t_lo >= t_hi) {  // (only with parts > 1)
        for (int r = tid; r < rows; r += 256) {
            stats[2 * r] = -INFINITY;
            stats[2 * r + 1] = 0.f;
        }
        return;
    }
    const int chunks = D / 8;  // 16-byte pieces of a row
    for (int idx = tid; idx < ROWS * chunks; idx += 256) {
        const int r = idx / chunks, c = idx - r * chunks;
        lt_cp16(Qs + (size_t)r * LDK + c * 8, a.qa + (size_t)(row0 + (r < rows ? r : 0)) * D + c * 8, r < rows);
    }
    const int* table = a.block_tables + (size_t)seq * a.max_blocks;
    auto find_slots = [&](int t) {  // the cache rows of key tile t (-1: behind the context, or no page)
        if (tid < KT) {
            const int j = t * KT + tid;
            int slot = -1;
            if (t < t_hi && j < kv_end) {
                const int blk = j / a.page_size;
                const int page = blk < a.max_blocks ? table[blk] : -1;
                if (page < 0 || page >= a.num_pages)
                    cw_report(a.status, CW_ST_PAGE_RANGE, tok0, page);
                else
                    slot = page * a.page_size + j % a.page_size;
            }
            slot_s[(t & 1) * KT + tid] = slot;
        }
    };
    const int c_step = 256 % chunks, r_step = 256 / chunks;
    auto fetch = [&](int t) {  // tile t into its stage (zeros where there is no key)
        bf16* stage = Ks + (size_t)(t & 1) * KT * LDK;
        const int* slots = slot_s + (t & 1) * KT;
        for (int r = tid / chunks, c = tid % chunks; r < KT;) {
            const int slot = slots[r];
            lt_cp16(stage + (size_t)r * LDK + c * 8, a.cache + (size_t)(slot < 0 ? 0 : slot) * D + c * 8, slot >= 0);
            c += c_step;
            r += r_step;
            if (c >= chunks) {
                c -= chunks;
                ++r;
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    // scores: this warp's rows 16 mw + g and + 8, keys KT / KW kw ..
    const int mw = warp % MT, kw = warp / MT, g = lane >> 2, q4 = lane & 3;
    const int r0 = mw * 16 + g, r1 = r0 + 8;
    const int pos0 = p0 + (head0 + r0) / H, pos1 = p0 + (head0 + r1) / H;  // the positions of its two rows
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
    // second product: m-tiles MP rw .., columns of n-tiles first_nt ..
    const int rw = warp % L::RW, cw = warp / L::RW;
    const int ntiles = rank / 8, per_warp = (((ntiles + L::CW - 1) / L::CW) + 1) & ~1;  // (even: n-tiles are read in pairs)
    const int first_nt = cw * per_warp, my_nt = max(0, min(per_warp, ntiles - first_nt));
    float acc[L::MP][L::NP][4];
#pragma unroll
    for (int i = 0; i < L::MP; ++i)
#pragma unroll
        for (int n = 0; n < L::NP; ++n) acc[i][n][0] = acc[i][n][1] = acc[i][n][2] = acc[i][n][3] = 0.f;
    find_slots(t_lo);
    find_slots(t_lo + 1);
    __syncthreads();
    fetch(t_lo);
    for (int t = t_lo; t < t_hi; ++t) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();  // tile t has landed for everyone (and the queries, at the first), and everyone has left tile t - 1
        if (t + 1 < t_hi) fetch(t + 1);
        find_slots(t + 2);  // (tile t's own slots are used up: its fetch was issued before the barrier above)
        const bf16* Kt = Ks + (size_t)(t & 1) * KT * LDK;
        float s[NS][4];
#pragma unroll
        for (int n = 0; n < NS; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
        const bf16* qrow = Qs + (size_t)(mw * 16 + (lane & 15)) * LDK + (lane >> 4) * 8;
        const bf16* krow = Kt + (size_t)kw * NS * 8 * LDK;
#pragma unroll 4
        for (int kk = 0; kk < D; kk += 16) {
            unsigned qf[4];
            lt_ldm(qf, qrow + kk);
            if (NS >= 2) {
                unsigned kf[4];
                lt_ldm(kf, krow + (size_t)((lane & 7) + (lane >> 4) * 8) * LDK + kk + ((lane >> 3) & 1) * 8);
                lt_mma(s[0], qf, kf[0], kf[1]);
                lt_mma(s[NS >= 2 ? 1 : 0], qf, kf[2], kf[3]);
            }
            if (NS & 1) {
                unsigned kf[2];
                lt_ldm2(kf, krow + (size_t)((NS - 1) * 8 + (lane & 7)) * LDK + kk + ((lane >> 3) & 1) * 8);
                lt_mma(s[NS - 1], qf, kf[0], kf[1]);
            }
        }
        float top0 = -INFINITY, top1 = -INFINITY;
#pragma unroll
        for (int n = 0; n < NS; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int key = t * KT + (kw * NS + n) * 8 + q4 * 2 + (e & 1);
                s[n][e] = key <= (e < 2 ? pos0 : pos1) && (e < 2 ? r0 : r1) < rows ? s[n][e] * a.scale : -INFINITY;
                if (e < 2) top0 = fmaxf(top0, s[n][e]); else top1 = fmaxf(top1, s[n][e]);
            }
        top0 = fmaxf(top0, __shfl_xor_sync(0xffffffffu, top0, 1));
        top0 = fmaxf(top0, __shfl_xor_sync(0xffffffffu, top0, 2));
        top1 = fmaxf(top1, __shfl_xor_sync(0xffffffffu, top1, 1));
        top1 = fmaxf(top1, __shfl_xor_sync(0xffffffffu, top1, 2));
        if (q4 == 0) {
            row_max[kw * ROWS + r0] = top0;
            row_max[kw * ROWS + r1] = top1;
        }
        __syncthreads();
        float n0 = m0, n1 = m1;
#pragma unroll
        for (int w = 0; w < KW; ++w) {
            n0 = fmaxf(n0, row_max[w * ROWS + r0]);
            n1 = fmaxf(n1, row_max[w * ROWS + r1]);
        }
        float sum0 = 0.f, sum1 = 0.f;
#pragma unroll
        for (int n = 0; n < NS; ++n) {
            float p[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) p[e] = s[n][e] == -INFINITY ? 0.f : expf(s[n][e] - (e < 2 ? n0 : n1));
            sum0 += p[0] + p[1];
            sum1 += p[2] + p[3];
            bf16 hi[4], lo[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                hi[e] = __float2bfloat16_rn(p[e]);
                lo[e] = __float2bfloat16_rn(p[e] - __bfloat162float(hi[e]));
            }
            const int col = (kw * NS + n) * 8 + q4 * 2;
            *(unsigned*)(Phi + r0 * PLD + col) = lt_pack(hi[0], hi[1]);
            *(unsigned*)(Phi + r1 * PLD + col) = lt_pack(hi[2], hi[3]);
            *(unsigned*)(Plo + r0 * PLD + col) = lt_pack(lo[0], lo[1]);
            *(unsigned*)(Plo + r1 * PLD + col) = lt_pack(lo[2], lo[3]);
        }
        sum0 += __shfl_xor_sync(0xffffffffu, sum0, 1);
        sum0 += __shfl_xor_sync(0xffffffffu, sum0, 2);
        sum1 += __shfl_xor_sync(0xffffffffu, sum1, 1);
        sum1 += __shfl_xor_sync(0xffffffffu, sum1, 2);
        const float f0 = m0 == -INFINITY ? 0.f : expf(m0 - n0), f1 = m1 == -INFINITY ? 0.f : expf(m1 - n1);
        if (q4 == 0) {
            row_sum[kw * ROWS + r0] = sum0;
            row_sum[kw * ROWS + r1] = sum1;
            if (kw == 0) {
                alpha_s[r0] = f0;
                alpha_s[r1] = f1;
            }
        }
        m0 = n0;
        m1 = n1;
        __syncthreads();
        float t0 = 0.f, t1 = 0.f;
#pragma unroll
        for (int w = 0; w < KW; ++w) {  // in warp order: the same sum in every thread
            t0 += row_sum[w * ROWS + r0];
            t1 += row_sum[w * ROWS + r1];
        }
        l0 = l0 * f0 + t0;
        l1 = l1 * f1 + t1;
        // weights times this warp's columns of the cached tile
#pragma unroll
        for (int i = 0; i < L::MP; ++i) {
            const float u0 = alpha_s[(rw * L::MP + i) * 16 + g], u1 = alpha_s[(rw * L::MP + i) * 16 + g + 8];
#pragma unroll
            for (int n = 0; n < L::NP; ++n) {
                acc[i][n][0] *= u0;
                acc[i][n][1] *= u0;
                acc[i][n][2] *= u1;
                acc[i][n][3] *= u1;
            }
        }
#pragma unroll
        for (int ks = 0; ks < KT / 16; ++ks) {
            unsigned ah[L::MP][4], al[L::MP][4];
#pragma unroll
            for (int i = 0; i < L::MP; ++i) {
                const int at = ((rw * L::MP + i) * 16 + (lane & 15)) * PLD + ks * 16 + (lane >> 4) * 8;
                lt_ldm(ah[i], Phi + at);
                lt_ldm(al[i], Plo + at);
            }
#pragma unroll
            for (int np = 0; np < L::NP / 2; ++np) {
                if (np * 2 < my_nt) {
                    unsigned b[4];
                    lt_ldm_t(b, Kt + (size_t)(ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LDK + (first_nt + np * 2) * 8 + (lane >> 4) * 8);
#pragma unroll
                    for (int i = 0; i < L::MP; ++i) {
                        lt_mma(acc[i][np * 2], ah[i], b[0], b[1]);
                        lt_mma(acc[i][np * 2 + 1], ah[i], b[2], b[3]);  // (an odd count's last pair also fills a tile that is not stored)
                    }
#pragma unroll
                    for (int i = 0; i < L::MP; ++i) {
                        lt_mma(acc[i][np * 2], al[i], b[0], b[1]);
                        lt_mma(acc[i][np * 2 + 1], al[i], b[2], b[3]);
                    }
                }
            }
        }
    }
    if (kw == 0 && q4 == 0) {
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int r = half ? r1 : r0;
            const float m = half ? m1 : m0, l = half ? l1 : l0;
            if (a.parts > 1) {
                inv_s[r] = 1.f;
                if (r < rows) {
                    stats[2 * r] = m;
                    stats[2 * r + 1] = l;
                }
            } else {  // the sink joins the denominator only
                const float sk = a.sink != nullptr ? a.sink[(head0 + r) % H] : -INFINITY;
                const float top = fmaxf(m, sk);
                const float keep = m == -INFINITY ? 0.f : expf(m - top);
                const float denom = l * keep + (sk == -INFINITY ? 0.f : expf(sk - top));
                inv_s[r] = denom > 0.f ? keep / denom : 0.f;
            }
        }
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < L::MP; ++i)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int r = (rw * L::MP + i) * 16 + g + half * 8;
            if (r >= rows) continue;
            const float inv = inv_s[r];
#pragma unroll
            for (int n = 0; n < L::NP; ++n)
                if (n < my_nt) {
                    const int col = (first_nt + n) * 8 + q4 * 2;
                    const float x = acc[i][n][half * 2] * inv, y = acc[i][n][half * 2 + 1] * inv;
                    if (a.parts > 1)
                        *(float2*)(sums + (size_t)r * rank + col) = make_float2(x, y);
                    else
                        *(unsigned*)(a.out + (size_t)(row0 + r) * rank + col) = lt_pack(__float2bfloat16_rn(x), __float2bfloat16_rn(y));
                }
        }
}

// The parts of a row's keys, added up in part order: a block per row, a thread per pair of columns.  The statistics' float2
// loads need partial at 8-byte boundaries: parts * rows * rank is even since the rank is a multiple of 8.
__global__ void __launch_bounds__(256)
latent_merge_kernel(const float* __restrict__ partial, const int* __restrict__ tok_seq, const float* __restrict__ sink,
                    bf16* __restrict__ out, int H, int rank, int parts, long long total_rows) {
    __shared__ float factor[LT_MAX_PARTS];
    pdl_wait();
    const long long row = blockIdx.x;
    if (tok_seq[row / H] < 0) return;  // (the attention kernel wrote the zeros)
    const float* stats = partial + (size_t)parts * total_rows * rank;
    const int lane = threadIdx.x & 31;
    float ms[LT_MAX_PARTS / 32], ls[LT_MAX_PARTS / 32], m = -INFINITY, l = 0.f;  // every warp looks at all parts, a lane at every 32nd
#pragma unroll
    for (int i = 0; i < LT_MAX_PARTS / 32; ++i) {
        const int s = i * 32 + lane;
        const float2 v = s < parts ? *(const float2*)(stats + ((size_t)s * total_rows + row) * 2) : make_float2(-INFINITY, 0.f);
        ms[i] = v.x;
        ls[i] = v.y;
        m = fmaxf(m, v.x);
    }
    const float sk = sink != nullptr ? sink[row % H] : -INFINITY;
    m = fmaxf(warp_max(m), sk);
#pragma unroll
    for (int i = 0; i < LT_MAX_PARTS / 32; ++i) {
        const float f = ms[i] == -INFINITY ? 0.f : expf(ms[i] - m);
        l = fmaf(f, ls[i], l);
        if (threadIdx.x < 32) factor[i * 32 + lane] = f;
    }
    l = warp_sum(l) + (sk == -INFINITY ? 0.f : expf(sk - m));
    __syncthreads();
    const float inv = l > 0.f ? 1.f / l : 0.f;
    for (int c = threadIdx.x * 2; c < rank; c += blockDim.x * 2) {
        float x = 0.f, y = 0.f;
        for (int s0 = 0; s0 < parts; s0 += 8) {  // eight parts' loads in flight together
            float2 v[8];
            float f[8];
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                f[i] = s0 + i < parts ? factor[s0 + i] : 0.f;
                v[i] = make_float2(0.f, 0.f);  // (a part without keys left no sums)
                if (f[i] != 0.f) v[i] = *(const float2*)(partial + ((size_t)(s0 + i) * total_rows + row) * rank + c);
            }
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                x = fmaf(f[i], v[i].x, x);
                y = fmaf(f[i], v[i].y, y);
            }
        }
        *(unsigned*)(out + row * rank + c) = lt_pack(__float2bfloat16_rn(x * inv), __float2bfloat16_rn(y * inv));
    }
}

static int g_latent_mma = 1;
extern "C" int cw_latent_attention_set_mma(int on) { g_latent_mma = on ? 1 : 0; return CW_OK; }

template <int MT>
static int launch_latent_mma(const LatentArgs& a, cudaStream_t stream) {
    using L = LatentTile<MT>;
    const size_t bytes = L::smem(a.rank + a.rot);
    static size_t allowed = 48 << 10;
    if (bytes > allowed) {
        const cudaError_t e = cudaFuncSetAttribute(latent_attention_mma_kernel<MT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
        if (e != cudaSuccess) return (int)e;
        allowed = bytes;
    }
    const long long rows = (long long)a.N * a.H;
    const dim3 grid((unsigned)((rows + L::ROWS - 1) / L::ROWS + a.S), a.parts);
    const int rc = cw_launch_ordered(latent_attention_mma_kernel<MT>, grid, dim3(256), bytes, stream, a);
    if (rc != 0 || a.parts == 1) return rc;
    int threads = 32;
    while (threads < 256 && threads * 2 < a.rank) threads *= 2;
    return cw_launch_ordered(latent_merge_kernel, dim3((unsigned)rows), dim3(threads), 0, stream, (const float*)a.partial, a.tok_seq, a.sink,
                             a.out, a.H, a.rank, a.parts, rows);
}

// Whether bfloat16 calls of these sizes run on the tensor cores (and may cut the keys in parts).
extern "C" int cw_latent_attention_on_tensor_cores(int rank, int rot) {
    const int D = rank + rot;
    return g_latent_mma && D % 16 == 0 && rank % 8 == 0 && rank <= 512 && D <= 640;
}

// few_rows: single tokens, or portions so short that a tile of 64 rows would be mostly empty.  parts > 1: `partial` holds
// parts * N * H * (rank + 2) floats.
extern "C" int cw_latent_attention(const void* qa, void* out, const void* cache, const int* block_tables, const int* tok_seq,
                                   const int* positions, const int* q_start, int S, const float* sink, int N, int H, int rank, int rot,
                                   int page_size, int max_blocks, int num_pages, float scale, int few_rows, int parts, float* partial,
                                   int dtype, int* status, cudaStream_t stream) {
    if (N == 0) return CW_OK;
    if (N < 0 || H <= 0 || rank <= 0 || rot < 0 || page_size <= 0 || max_blocks <= 0 || S <= 0 || q_start == nullptr) return CW_ERR_BAD_SIZE;
    if (parts < 1 || parts > LT_MAX_PARTS || (parts > 1 && partial == nullptr)) return CW_ERR_BAD_SIZE;
    if (dtype == 1 && cw_latent_attention_on_tensor_cores(rank, rot) && (long long)N * H <= 0x3fffffffLL && ((uintptr_t)qa & 15) == 0 &&
        ((uintptr_t)cache & 15) == 0 && ((uintptr_t)out & 3) == 0) {
        const LatentArgs args = {(const bf16*)qa, (bf16*)out, (const bf16*)cache, block_tables, tok_seq, positions, q_start, sink, N, S, H,
                                 rank, rot, page_size, max_blocks, num_pages, scale, parts, partial, status};
        return few_rows ? launch_latent_mma<1>(args, stream) : launch_latent_mma<4>(args, stream);
    }
    if (rank > LA_CH * LA_NC || (H + LA_HB - 1) / LA_HB > 65535) return CW_ERR_UNSUPPORTED;
    const size_t smem = (size_t)LA_HB * (rank + rot) * sizeof(float);
    dim3 grid(N, (H + LA_HB - 1) / LA_HB);
    if (dtype == 0)
        return cw_launch_ordered(latent_attention_kernel<float, float>, grid, dim3(LA_CH), smem, stream, (const float*)qa, (float*)out,
                         (const float*)cache, block_tables, tok_seq, positions, sink, H, rank, rot, page_size, max_blocks,
                         num_pages, scale, status);
    if (dtype == 1)
        return cw_launch_ordered(latent_attention_kernel<bf16, bf16>, grid, dim3(LA_CH), smem, stream, (const bf16*)qa, (bf16*)out,
                         (const bf16*)cache, block_tables, tok_seq, positions, sink, H, rank, rot, page_size, max_blocks,
                         num_pages, scale, status);
    return CW_ERR_BAD_DTYPE;
}

CW_TRACE_TU(latent_attention)
