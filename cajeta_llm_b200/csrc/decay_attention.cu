// Linear attention with one constant decay per head:
//
//     S_t = lambda_h S_(t-1) + k_t v_t^T ;  o_t = S_t^T q_t            (S: dim x vdim, float32, zero at the start)
//
// A request's S matrices live in its slot of the state tensor, [heads][dim][vdim] float32 row by row.  A step's rows
// are laid out request after request (req_start, req_slot: device metadata only, so steps can be captured); a request
// that a captured step is filled up with (slot -1, no rows) is left alone.
//
//   walk     every token in order: the state's rows dealt to eight warps, its columns to their lanes, all of it in
//            registers; single decoded tokens, short portions, and everything on the 32-bit path
//            (the next tokens' inputs are on their way to registers while these are walked)
//   chunk    (bfloat16 q, k, v) portions of a prompt, 64 tokens at a time on the tensor cores:
//                O = (Q K^T . L) V + diag(lambda^(i+1)) Q S ,   L_ij = lambda^(i-j) for j <= i, else 0
//                S <- lambda^n S + K^T diag(lambda^(n-1-j)) V
//            A portion is cut into segments that run side by side: a first kernel works out what each segment adds to
//            the state (the last line alone, from zero), a second one starts every segment from the state it begins with,
//            lambda^(start) S_0 + sum over the segments before it (S_0 read from a copy that the first kernel made: the
//            request's last segment writes the state while others may not have begun).
//   gated_row_norm   o / rms(o) * w * sigmoid(g), one norm over a whole row (all heads side by side)
//
// Precision: the state and its decays are float32 throughout; q, k and v are what the projection left (bfloat16 on the
// bfloat16 path).  Where a float32 value enters a bfloat16 product - the scores Q K^T . L, the state under the queries, the
// decayed values - it goes in as two bfloat16 terms (its value to 2^-17), summed in float32.
#define CJ_LIB "decay_attention"
#include "common.cuh"

using namespace cj;

namespace {

// ---------------------------------------------------------------------------------
// walk
// ---------------------------------------------------------------------------------
struct WalkArgs {
    const void* x;                // [T, ld]: q | k | v at columns off_q, off_k, off_v, head by head
    int ld, off_q, off_k, off_v;
    const float* decay;           // [heads]
    float* state;
    long long slot_stride;
    const int* req_start;
    const int* req_slot;
    float* out;                   // [T, heads * vdim]
    int heads, dim, vdim;
    int most;                     // requests with more rows than this are left to the chunk kernels (0: none are)
};

constexpr int WALK_WARPS = 8, WALK_TOK = 8;

// A block: one request, one head, 32 columns of the state.  Warp w holds rows w, w + 8, ...: ROWS of them.
template <typename TX, int ROWS>
__global__ void __launch_bounds__(WALK_WARPS * 32) walk_kernel(WalkArgs p) {
    cj::after_predecessor();
    cj::release_successor();
    constexpr int DIM = ROWS * WALK_WARPS;
    __shared__ __align__(16) float qs[WALK_TOK][DIM], ks[WALK_TOK][DIM];        // entry d lies at (d % 8) * ROWS + d / 8
    __shared__ float vs[WALK_TOK][32];
    __shared__ float part[WALK_TOK][WALK_WARPS][32];
    const int req = blockIdx.x, head = blockIdx.y;
    const int slot = p.req_slot[req];
    const int first = p.req_start[req], n = p.req_start[req + 1] - first;
    if (slot < 0 || n <= 0 || (p.most > 0 && n > p.most)) return;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int col = blockIdx.z * 32 + lane;
    const bool live = col < p.vdim;
    float* S = p.state + (size_t)slot * p.slot_stride + (size_t)head * p.dim * p.vdim;
    float s[ROWS];
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
        const int d = warp + WALK_WARPS * i;
        s[i] = live && d < p.dim ? S[(size_t)d * p.vdim + col] : 0.0f;
    }
    const float decay = p.decay[head];
    // what this thread brings of WALK_TOK tokens: entries thread + 256 i of their [WALK_TOK][DIM] queries and keys, one value
    constexpr int MINE = WALK_TOK * DIM / (WALK_WARPS * 32);
    static_assert(MINE >= 1 && WALK_TOK == WALK_WARPS, "a block's threads share out the tokens' entries evenly");
    float q_next[MINE], k_next[MINE], v_next;
    auto fetch = [&](int t0) {
        const TX* base = (const TX*)p.x + (size_t)(first + t0) * p.ld;
#pragma unroll
        for (int i = 0; i < MINE; ++i) {
            const int e = threadIdx.x + WALK_WARPS * 32 * i, t = e / DIM, d = e % DIM;
            const bool ok = t0 + t < n && d < p.dim;
            const TX* row = base + (size_t)(ok ? t : 0) * p.ld + head * p.dim + (ok ? d : 0);
            q_next[i] = ok ? to_f32(row[p.off_q]) : 0.0f;
            k_next[i] = ok ? to_f32(row[p.off_k]) : 0.0f;
        }
        const bool ok = t0 + warp < n && live;
        v_next = ok ? to_f32(base[(size_t)warp * p.ld + p.off_v + head * p.vdim + col]) : 0.0f;
    };
    fetch(0);
    for (int t0 = 0; t0 < n; t0 += WALK_TOK) {
        const int nt = min(WALK_TOK, n - t0);
#pragma unroll
        for (int i = 0; i < MINE; ++i) {
            const int e = threadIdx.x + WALK_WARPS * 32 * i, t = e / DIM, d = e % DIM;
            const int at = (d % WALK_WARPS) * ROWS + d / WALK_WARPS;
            qs[t][at] = q_next[i];
            ks[t][at] = k_next[i];
        }
        vs[warp][lane] = v_next;
        __syncthreads();
        if (t0 + WALK_TOK < n) fetch(t0 + WALK_TOK);
        for (int t = 0; t < nt; ++t) {
            const float v = vs[t][lane];
            const float4* k4 = (const float4*)(ks[t] + warp * ROWS);
            const float4* q4 = (const float4*)(qs[t] + warp * ROWS);
            float y = 0.0f;
#pragma unroll
            for (int i = 0; i < ROWS; i += 4) {
                const float4 k = k4[i / 4], q = q4[i / 4];
                s[i] = fmaf(decay, s[i], k.x * v);
                s[i + 1] = fmaf(decay, s[i + 1], k.y * v);
                s[i + 2] = fmaf(decay, s[i + 2], k.z * v);
                s[i + 3] = fmaf(decay, s[i + 3], k.w * v);
                y = fmaf(s[i], q.x, y);
                y = fmaf(s[i + 1], q.y, y);
                y = fmaf(s[i + 2], q.z, y);
                y = fmaf(s[i + 3], q.w, y);
            }
            part[t][warp][lane] = y;
        }
        __syncthreads();
        for (int t = warp; t < nt; t += WALK_WARPS) {
            float y = 0.0f;
#pragma unroll
            for (int w = 0; w < WALK_WARPS; ++w) y += part[t][w][lane];
            if (live) p.out[(size_t)(first + t0 + t) * p.heads * p.vdim + head * p.vdim + col] = y;
        }
        // the next round's staging writes only what everyone has read; its sums are written after its first barrier
    }
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
        const int d = warp + WALK_WARPS * i;
        if (live && d < p.dim) S[(size_t)d * p.vdim + col] = s[i];
    }
}

// ---------------------------------------------------------------------------------
// chunk
// ---------------------------------------------------------------------------------
__device__ __forceinline__ void cp_async16(void* smem, const void* gmem, bool valid) {
    unsigned s = (unsigned)__cvta_generic_to_shared(smem);
    int n = valid ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(s), "l"(gmem), "r"(n) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

__device__ __forceinline__ void ldmatrix_x4(unsigned (&r)[4], const void* smem) {
    unsigned s = (unsigned)__cvta_generic_to_shared(smem);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(s));
}
__device__ __forceinline__ void ldmatrix_x4_trans(unsigned (&r)[4], const void* smem) {
    unsigned s = (unsigned)__cvta_generic_to_shared(smem);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(s));
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ unsigned pack_bf16(float lo, float hi) {
    __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *(unsigned*)&v;
}
__device__ __forceinline__ float low_f32(unsigned v) { return __uint_as_float(v << 16); }
__device__ __forceinline__ float high_f32(unsigned v) { return __uint_as_float(v & 0xffff0000u); }
// two float32 values as a bfloat16 pair and the pair of what it leaves over
__device__ __forceinline__ void split_pair(float lo, float hi, unsigned& first, unsigned& rest) {
    first = pack_bf16(lo, hi);
    rest = pack_bf16(lo - low_f32(first), hi - high_f32(first));
}
// element (row, col) of a [rows][W] bf16 tile whose 16-byte pieces are XOR-swizzled by row (W a multiple of 64)
template <int W>
__device__ __forceinline__ __nv_bfloat16* tile_ptr(__nv_bfloat16* base, int row, int col) {
    return base + row * W + (((col >> 3) ^ (row & 7)) << 3) + (col & 7);
}

constexpr int CHUNK = 64;

struct ChunkArgs {
    const __nv_bfloat16* x;
    int ld, off_q, off_k, off_v;
    const float* powers;          // [heads][CHUNK + 1]: lambda^0 .. lambda^CHUNK
    const double* log2_decay;     // [heads]
    float* state;
    long long slot_stride;
    const int* req_start;
    const int* req_slot;
    int n_requests;
    float* out;                   // [T, heads * vdim]
    float4* added;                // [segments][heads][column tiles][D / 8][threads]: what a segment adds to the state, in the order the
                                  // threads hold it; in a request's last one S_0
    int heads, dim, vdim;
    int seg;                      // tokens of a segment (a multiple of CHUNK)
    int most;                     // requests of at most this many rows are left to the walk
};

// lambda^n for the distances between segments
__device__ __forceinline__ float power_of(double log2_decay, int n) { return n == 0 ? 1.0f : (float)exp2(log2_decay * (double)n); }

template <int D, int WARPS>
struct ChunkSmem {
    static constexpr int V = 16 * WARPS;                     // state columns of a block
    static constexpr int STAGE = CHUNK * (2 * D + V);        // bf16 entries of one chunk's q, k and v
    static constexpr int BYTES = (2 * STAGE + 2 * CHUNK * CHUNK) * 2 + (CHUNK + 1) * 4;
};

// A block: one segment of one request, one head, 16 WARPS columns of the state; warp w holds S^T rows 16 w .. 16 w + 15
// (columns of the state) as a float32 accumulator over all D of its rows.
// ADDED: only what the segment adds to the state, starting from zero, stored in `added` (not for a request's last segment).
template <int D, int WARPS, bool ADDED>
__global__ void __launch_bounds__(32 * WARPS) chunk_kernel(ChunkArgs p) {
    cj::after_predecessor();
    cj::release_successor();
    using Sm = ChunkSmem<D, WARPS>;
    constexpr int V = Sm::V, THREADS = 32 * WARPS;
    extern __shared__ __align__(128) unsigned char smem_raw[];
    __nv_bfloat16* stage0 = (__nv_bfloat16*)smem_raw;
    __nv_bfloat16* p_hi = stage0 + 2 * Sm::STAGE;            // [CHUNK][CHUNK]: the decayed scores' two terms
    __nv_bfloat16* p_lo = p_hi + CHUNK * CHUNK;
    float* pw = (float*)(p_lo + CHUNK * CHUNK);              // [CHUNK + 1]

    // which request and which of its segments
    int at = blockIdx.x, req = -1, lo = 0, n_all = 0, n_segs = 0;
    for (int r = 0; r < p.n_requests; ++r) {
        const int a = p.req_start[r], n = p.req_start[r + 1] - a;
        if (n <= p.most || p.req_slot[r] < 0) continue;
        const int segs = (n + p.seg - 1) / p.seg;
        if (at < segs) { req = r; lo = a; n_all = n; n_segs = segs; break; }
        at -= segs;
    }
    if (req < 0) return;
    const int s0 = at * p.seg;                               // the segment's first token within the portion
    const int n = min(p.seg, n_all - s0);
    const bool last = s0 + n == n_all;
    if (ADDED && last) return;
    const int head = blockIdx.y, v0 = blockIdx.z * V;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int g = lane >> 2, t4 = lane & 3, mi = lane >> 3;
    const int first = lo + s0;

    auto fetch = [&](int c0, __nv_bfloat16* st) {
        const int rows = min(CHUNK, n - c0);
        constexpr int CD = D / 8, CV = V / 8;
        for (int i = tid; i < CHUNK * CD; i += THREADS) {
            const int r = i / CD, c = i % CD;
            const bool ok = r < rows && c * 8 < p.dim;
            const __nv_bfloat16* row = p.x + (size_t)(first + c0 + (ok ? r : 0)) * p.ld + head * p.dim + (ok ? c * 8 : 0);
            if (!ADDED) cp_async16(st + r * D + ((c ^ (r & 7)) << 3), row + p.off_q, ok);
            cp_async16(st + CHUNK * D + r * D + ((c ^ (r & 7)) << 3), row + p.off_k, ok);
        }
        for (int i = tid; i < CHUNK * CV; i += THREADS) {
            const int r = i / CV, c = i % CV;
            const bool ok = r < rows && v0 + c * 8 < p.vdim;
            const __nv_bfloat16* row = p.x + (size_t)(first + c0 + (ok ? r : 0)) * p.ld + p.off_v + head * p.vdim + (ok ? v0 + c * 8 : 0);
            cp_async16(st + 2 * CHUNK * D + r * V + ((c ^ (r & 7)) << 3), row, ok);
        }
    };
    fetch(0, stage0);
    cp_async_commit();
    for (int i = tid; i <= CHUNK; i += THREADS) pw[i] = p.powers[(size_t)head * (CHUNK + 1) + i];

    // element (row d, column v) of the head's state, wherever a [dim][vdim] matrix of it lies
    const int va = v0 + warp * 16 + g, vb = va + 8;          // this thread's two columns of the state
    float S[D / 8][4];                                       // S^T: [j][0,1] = (va, 8 j + 2 t4 + 0,1), [2,3] = (vb, ..)
#pragma unroll
    for (int j = 0; j < D / 8; ++j) S[j][0] = S[j][1] = S[j][2] = S[j][3] = 0.0f;
    float* state = p.state + (size_t)p.req_slot[req] * p.slot_stride + (size_t)head * p.dim * p.vdim;
    auto state_at = [&](int j, int e, bool& ok) {            // where entry e of S[j] lies in a [dim][vdim] matrix
        const int d = 8 * j + 2 * t4 + (e & 1), v = e < 2 ? va : vb;
        ok = d < p.dim && v < p.vdim;
        return ok ? (size_t)d * p.vdim + v : (size_t)0;
    };
    auto read_state = [&]() {
#pragma unroll
        for (int j = 0; j < D / 8; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                bool ok;
                const float v = state[state_at(j, e, ok)];
                S[j][e] = ok ? v : 0.0f;
            }
    };
    auto held = [&](int segment) {                           // this thread's part of what the launch's segment left in `added`
        return p.added + (((size_t)segment * p.heads + head) * gridDim.z + blockIdx.z) * (D / 8) * THREADS + tid;
    };
    auto keep_in = [&](float4* m) {
#pragma unroll
        for (int j = 0; j < D / 8; ++j) m[(size_t)j * THREADS] = make_float4(S[j][0], S[j][1], S[j][2], S[j][3]);
    };
    if (ADDED && at == 0) {
        read_state();
        keep_in(held(blockIdx.x + n_segs - 1));
#pragma unroll
        for (int j = 0; j < D / 8; ++j) S[j][0] = S[j][1] = S[j][2] = S[j][3] = 0.0f;
    }
    if (!ADDED && n_segs == 1) read_state();
    if (!ADDED && n_segs > 1) {
        const double l2 = p.log2_decay[head];
        const int base = blockIdx.x - at;
        for (int s = -1; s < at; ++s) {
            // S_0, then the segments before this one: segment s ends (at - 1 - s) whole segments before this one begins
            const float4* m = held(s < 0 ? base + n_segs - 1 : base + s);
            const float f = power_of(l2, s < 0 ? s0 : (at - 1 - s) * p.seg);
#pragma unroll
            for (int j = 0; j < D / 8; ++j) {
                const float4 a = m[(size_t)j * THREADS];
                S[j][0] = fmaf(f, a.x, S[j][0]);
                S[j][1] = fmaf(f, a.y, S[j][1]);
                S[j][2] = fmaf(f, a.z, S[j][2]);
                S[j][3] = fmaf(f, a.w, S[j][3]);
            }
        }
    }

    int cur = 0;
    for (int c0 = 0; c0 < n; c0 += CHUNK, cur ^= 1) {
        if (c0 + CHUNK < n) fetch(c0 + CHUNK, stage0 + (cur ^ 1) * Sm::STAGE);
        cp_async_commit();
        cp_async_wait<1>();
        __syncthreads();
        __nv_bfloat16* qs = stage0 + cur * Sm::STAGE;
        __nv_bfloat16* ks = qs + CHUNK * D;
        __nv_bfloat16* vs = ks + CHUNK * D;
        const int nc = min(CHUNK, n - c0);
        if (!ADDED) {
            // decayed scores: WARPS / 4 warps share 16 query rows, each takes its columns
            constexpr int COLS = CHUNK * 4 / WARPS, NT = COLS / 8;
            const int i0 = (warp & 3) * 16, j0 = (warp >> 2) * COLS;
            float sc[NT][4];
#pragma unroll
            for (int j = 0; j < NT; ++j) sc[j][0] = sc[j][1] = sc[j][2] = sc[j][3] = 0.0f;
            if (j0 <= i0 + 15) {
#pragma unroll
                for (int kk = 0; kk < D / 16; ++kk) {
                    unsigned qf[4];
                    ldmatrix_x4(qf, tile_ptr<D>(qs, i0 + (lane & 15), kk * 16 + (lane >> 4) * 8));
#pragma unroll
                    for (int jp = 0; jp < NT / 2; ++jp) {
                        unsigned b[4];
                        ldmatrix_x4(b, tile_ptr<D>(ks, j0 + jp * 16 + (mi >> 1) * 8 + (lane & 7), kk * 16 + (mi & 1) * 8));
                        mma_bf16(sc[2 * jp], qf, b[0], b[1]);
                        mma_bf16(sc[2 * jp + 1], qf, b[2], b[3]);
                    }
                }
            }
#pragma unroll
            for (int j = 0; j < NT; ++j)
#pragma unroll
                for (int h = 0; h < 2; ++h) {
                    const int i = i0 + g + 8 * h, col = j0 + j * 8 + 2 * t4;
                    const float a = col <= i ? sc[j][2 * h] * pw[i - col] : 0.0f;
                    const float b = col + 1 <= i ? sc[j][2 * h + 1] * pw[i - col - 1] : 0.0f;
                    unsigned hi, rest;
                    split_pair(a, b, hi, rest);
                    *(unsigned*)tile_ptr<CHUNK>(p_hi, i, col) = hi;
                    *(unsigned*)tile_ptr<CHUNK>(p_lo, i, col) = rest;
                }
            // the state under the queries: O^T = S^T Q^T, then column i times lambda^(i + 1)
            float o[CHUNK / 8][4];
#pragma unroll
            for (int i = 0; i < CHUNK / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
#pragma unroll
            for (int kk = 0; kk < D / 16; ++kk) {
                unsigned hi[4], rest[4];
                split_pair(S[2 * kk][0], S[2 * kk][1], hi[0], rest[0]);
                split_pair(S[2 * kk][2], S[2 * kk][3], hi[1], rest[1]);
                split_pair(S[2 * kk + 1][0], S[2 * kk + 1][1], hi[2], rest[2]);
                split_pair(S[2 * kk + 1][2], S[2 * kk + 1][3], hi[3], rest[3]);
#pragma unroll
                for (int ip = 0; ip < CHUNK / 16; ++ip) {
                    unsigned b[4];
                    ldmatrix_x4(b, tile_ptr<D>(qs, ip * 16 + (mi >> 1) * 8 + (lane & 7), kk * 16 + (mi & 1) * 8));
                    mma_bf16(o[2 * ip], hi, b[0], b[1]);
                    mma_bf16(o[2 * ip], rest, b[0], b[1]);
                    mma_bf16(o[2 * ip + 1], hi, b[2], b[3]);
                    mma_bf16(o[2 * ip + 1], rest, b[2], b[3]);
                }
            }
#pragma unroll
            for (int i = 0; i < CHUNK / 8; ++i) {
                const float f0 = pw[i * 8 + 2 * t4 + 1], f1 = pw[i * 8 + 2 * t4 + 2];
                o[i][0] *= f0; o[i][1] *= f1;
                o[i][2] *= f0; o[i][3] *= f1;
            }
            __syncthreads();                                 // the scores are complete
            // plus V^T P^T: keys 16 kk .. only reach the rows from there on
#pragma unroll
            for (int kk = 0; kk < CHUNK / 16; ++kk) {
                unsigned vf[4];
                ldmatrix_x4_trans(vf, tile_ptr<V>(vs, kk * 16 + (mi >> 1) * 8 + (lane & 7), warp * 16 + (mi & 1) * 8));
#pragma unroll
                for (int ip = kk; ip < CHUNK / 16; ++ip) {
                    unsigned b[4], c[4];
                    ldmatrix_x4(b, tile_ptr<CHUNK>(p_hi, ip * 16 + (mi >> 1) * 8 + (lane & 7), kk * 16 + (mi & 1) * 8));
                    ldmatrix_x4(c, tile_ptr<CHUNK>(p_lo, ip * 16 + (mi >> 1) * 8 + (lane & 7), kk * 16 + (mi & 1) * 8));
                    mma_bf16(o[2 * ip], vf, b[0], b[1]);
                    mma_bf16(o[2 * ip], vf, c[0], c[1]);
                    mma_bf16(o[2 * ip + 1], vf, b[2], b[3]);
                    mma_bf16(o[2 * ip + 1], vf, c[2], c[3]);
                }
            }
            float* dst = p.out + (size_t)(first + c0) * p.heads * p.vdim + head * p.vdim;
            const size_t ldo = (size_t)p.heads * p.vdim;
#pragma unroll
            for (int i = 0; i < CHUNK / 8; ++i)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int t = i * 8 + 2 * t4 + (e & 1), v = e < 2 ? va : vb;
                    if (t < nc && v < p.vdim) dst[t * ldo + v] = o[i][e];
                }
        }
        // the state moves on: S^T <- lambda^nc S^T + (V^T diag(lambda^(nc - 1 - j))) K
        if (ADDED || last || c0 + CHUNK < n) {
            const float keep = pw[nc];
#pragma unroll
            for (int j = 0; j < D / 8; ++j) {
                S[j][0] *= keep; S[j][1] *= keep;
                S[j][2] *= keep; S[j][3] *= keep;
            }
#pragma unroll
            for (int kk = 0; kk < CHUNK / 16; ++kk) {
                if (kk * 16 >= nc) break;
                unsigned vf[4], hi[4], rest[4];
                ldmatrix_x4_trans(vf, tile_ptr<V>(vs, kk * 16 + (mi >> 1) * 8 + (lane & 7), warp * 16 + (mi & 1) * 8));
                const int j = nc - 1 - (kk * 16 + 2 * t4);   // the exponent of this thread's first token of the step
                const float w0 = j >= 0 ? pw[j] : 0.0f, w1 = j >= 1 ? pw[j - 1] : 0.0f;
                const float w8 = j >= 8 ? pw[j - 8] : 0.0f, w9 = j >= 9 ? pw[j - 9] : 0.0f;
                split_pair(low_f32(vf[0]) * w0, high_f32(vf[0]) * w1, hi[0], rest[0]);
                split_pair(low_f32(vf[1]) * w0, high_f32(vf[1]) * w1, hi[1], rest[1]);
                split_pair(low_f32(vf[2]) * w8, high_f32(vf[2]) * w9, hi[2], rest[2]);
                split_pair(low_f32(vf[3]) * w8, high_f32(vf[3]) * w9, hi[3], rest[3]);
#pragma unroll
                for (int dp = 0; dp < D / 16; ++dp) {
                    unsigned b[4];
                    ldmatrix_x4_trans(b, tile_ptr<D>(ks, kk * 16 + (mi & 1) * 8 + (lane & 7), dp * 16 + (mi >> 1) * 8));
                    mma_bf16(S[2 * dp], hi, b[0], b[1]);
                    mma_bf16(S[2 * dp], rest, b[0], b[1]);
                    mma_bf16(S[2 * dp + 1], hi, b[2], b[3]);
                    mma_bf16(S[2 * dp + 1], rest, b[2], b[3]);
                }
            }
        }
        __syncthreads();                                     // this chunk's tiles and scores are read before they are written again
    }
    if (ADDED) keep_in(held(blockIdx.x));
    else if (last) {
#pragma unroll
        for (int j = 0; j < D / 8; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                bool ok;
                const size_t to = state_at(j, e, ok);
                if (ok) state[to] = S[j][e];
            }
    }
}

// ---------------------------------------------------------------------------------
// out[r] = y[r] / rms(y[r]) * w * sigmoid(z[r]): a block a row
// ---------------------------------------------------------------------------------
template <typename TZ, typename TO>
__global__ void gated_row_norm_kernel(const float* __restrict__ y, int n, const TZ* __restrict__ z, int ld_z, const float* __restrict__ w,
                                      float eps, TO* __restrict__ out) {
    cj::after_predecessor();
    cj::release_successor();
    __shared__ float scratch[32];
    const float* yr = y + (size_t)blockIdx.x * n;
    const TZ* zr = z + (size_t)blockIdx.x * ld_z;
    float ss = 0.0f;
    for (int i = threadIdx.x; i < n; i += blockDim.x) ss = fmaf(yr[i], yr[i], ss);
    ss = warp_sum(ss);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    if (lane == 0) scratch[warp] = ss;
    __syncthreads();
    float total = 0.0f;
    for (int i = 0; i < nw; ++i) total += scratch[i];
    const float scale = 1.0f / sqrtf(total / (float)n + eps);
    for (int i = threadIdx.x; i < n; i += blockDim.x)
        out[(size_t)blockIdx.x * n + i] = from_f32<TO>(yr[i] * scale * w[i] / (1.0f + expf(-to_f32(zr[i]))));
}

}  // namespace

// x: rows with stride ld in x_dtype; q, k, v at columns off_q, off_k, off_v (heads x dim, heads x dim, heads x vdim).
// decay: float32 [heads].  state: per slot heads x dim x vdim float32 from the given pointer on, slot_stride apart.
// most > 0: requests with more rows than that are left alone.  out: float32 [T, heads * vdim].
CJ_EXPORT int cj_decay_walk(const void* x, int x_dtype, int ld, int off_q, int off_k, int off_v, const float* decay, float* state,
                            long long slot_stride, const int* req_start, const int* req_slot, int requests, float* out, int heads,
                            int dim, int vdim, int most, cudaStream_t stream) {
    if (requests <= 0) return 0;
    if (!x || !decay || !state || !req_start || !req_slot || !out) return CJ_ERR_ARG;
    if (heads <= 0 || heads > 65535 || dim <= 0 || dim > 256 || vdim <= 0 || slot_stride < (long long)heads * dim * vdim) return CJ_ERR_SIZE;
    WalkArgs p{x, ld, off_q, off_k, off_v, decay, state, slot_stride, req_start, req_slot, out, heads, dim, vdim, most};
    const dim3 grid(requests, heads, (vdim + 31) / 32);
    if (grid.z > 65535) return CJ_ERR_SIZE;
#define LAUNCH(TX)                                                                                                      \
    do {                                                                                                                \
        if (dim <= 32) cj::launch(walk_kernel<TX, 4>, grid, dim3(WALK_WARPS * 32), 0, stream, p);                       \
        else if (dim <= 64) cj::launch(walk_kernel<TX, 8>, grid, dim3(WALK_WARPS * 32), 0, stream, p);                  \
        else if (dim <= 128) cj::launch(walk_kernel<TX, 16>, grid, dim3(WALK_WARPS * 32), 0, stream, p);                \
        else cj::launch(walk_kernel<TX, 32>, grid, dim3(WALK_WARPS * 32), 0, stream, p);                                \
    } while (0)
    if (x_dtype == CJ_F32) LAUNCH(float);
    else if (x_dtype == CJ_BF16) LAUNCH(__nv_bfloat16);
    else return CJ_ERR_DTYPE;
#undef LAUNCH
    return launch_status();
}

// The tensor-core form for requests with more rows than `most`.  x bfloat16, 16-byte aligned rows and columns; dim <= 128, dim and
// vdim multiples of 8.  seg: tokens of a segment, a multiple of 64; segments: blocks laid out for them, at least
// rows / seg + requests; added: scratch of cj_decay_added_floats float32 a segment, 16-byte aligned (may be null when
// every request fits one segment).
CJ_EXPORT int cj_decay_chunk(const void* x, int ld, int off_q, int off_k, int off_v, const float* powers, const double* log2_decay,
                             float* state, long long slot_stride, const int* req_start, const int* req_slot, int requests, float* out,
                             float* added, int segments, int heads, int dim, int vdim, int seg, int most, cudaStream_t stream) {
    if (requests <= 0 || segments <= 0) return 0;
    if (!x || !powers || !log2_decay || !state || !req_start || !req_slot || !out) return CJ_ERR_ARG;
    if (heads <= 0 || heads > 65535 || dim <= 0 || dim > 128 || vdim <= 0 || seg <= 0 || seg % CHUNK != 0 || most < 0) return CJ_ERR_SIZE;
    if (slot_stride < (long long)heads * dim * vdim) return CJ_ERR_SIZE;
    if ((dim | vdim | ld | off_q | off_k | off_v) % 8 != 0 || (((uintptr_t)x | (uintptr_t)added) & 15)) return CJ_ERR_ALIGN;
    ChunkArgs p{(const __nv_bfloat16*)x, ld, off_q, off_k, off_v, powers, log2_decay, state, slot_stride, req_start, req_slot, requests,
                out, (float4*)added, heads, dim, vdim, seg, most};
#define LAUNCH_ONE(D_, W_, A_)                                                                                          \
    do {                                                                                                                \
        constexpr int bytes = ChunkSmem<D_, W_>::BYTES;                                                                 \
        static bool sized = false;                                                                                      \
        if (!sized) {                                                                                                   \
            cudaError_t e = cudaFuncSetAttribute(chunk_kernel<D_, W_, A_>, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes); \
            if (e != cudaSuccess) return (int)e;                                                                        \
            sized = true;                                                                                               \
        }                                                                                                               \
        cj::launch(chunk_kernel<D_, W_, A_>, dim3(segments, heads, (vdim + 16 * W_ - 1) / (16 * W_)), dim3(32 * W_), bytes, stream, p); \
    } while (0)
#define LAUNCH(D_, W_)                                                                                                  \
    do {                                                                                                                \
        if (added) LAUNCH_ONE(D_, W_, true);                                                                            \
        LAUNCH_ONE(D_, W_, false);                                                                                      \
    } while (0)
    if (dim <= 64) { if (vdim <= 64) LAUNCH(64, 4); else LAUNCH(64, 8); }
    else { if (vdim <= 64) LAUNCH(128, 4); else LAUNCH(128, 8); }
#undef LAUNCH
#undef LAUNCH_ONE
    return launch_status();
}

// float32 entries of `added` that one segment needs
CJ_EXPORT long long cj_decay_added_floats(int heads, int dim, int vdim) {
    const int D = dim <= 64 ? 64 : 128, W = vdim <= 64 ? 4 : 8;
    return (long long)heads * ((vdim + 16 * W - 1) / (16 * W)) * (D / 8) * 4 * 32 * W;
}

// z: the gates' columns, rows ld_z apart, in z_dtype; (z, out): (float32, float32) or (bfloat16, bfloat16)
CJ_EXPORT int cj_gated_row_norm(const float* y, int n, const void* z, int z_dtype, int ld_z, const float* w, float eps, void* out,
                                int out_dtype, int rows, cudaStream_t stream) {
    if (rows <= 0) return 0;
    if (!y || !z || !w || !out || n <= 0) return CJ_ERR_ARG;
    if (z_dtype != out_dtype) return CJ_ERR_DTYPE;
    const int threads = n >= 2048 ? 512 : (n >= 512 ? 256 : 128);
    if (out_dtype == CJ_F32) cj::launch(gated_row_norm_kernel<float, float>, dim3(rows), dim3(threads), 0, stream, y, n, (const float*)z, ld_z, w, eps, (float*)out);
    else if (out_dtype == CJ_BF16) cj::launch(gated_row_norm_kernel<__nv_bfloat16, __nv_bfloat16>, dim3(rows), dim3(threads), 0, stream, y, n, (const __nv_bfloat16*)z, ld_z, w, eps, (__nv_bfloat16*)out);
    else return CJ_ERR_DTYPE;
    return launch_status();
}
