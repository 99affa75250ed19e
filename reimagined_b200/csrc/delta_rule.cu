// The generalized delta rule (per head: S <- diag(w) S - (a*u)(u^T S) + k v^T, o = S^T r) with its decays, removal
// rates, unit keys, head norm and output gate.  Everything here is fp32; states are stored [head][value][key].
//
// A value column j of a state evolves on its own:  s_j <- w*s_j + (k v_j - (a*u) (u.s_j)),  o_j = r.s_j,  so the
// columns are spread over threads and CTAs and only the dot products over the keys cross lanes: eight or sixteen lanes
// share a column, each holding its groups of four keys in registers, and the arithmetic runs on packed fp32 pairs.
//
//   delta_scan_kernel   a sequence of tokens, two per round: a CTA owns 32 columns of a head.  Eight producer warps turn
//                       the raw projections of the next sixteen tokens into records in shared memory while four
//                       consumer warps walk the current ones with the state in registers.
//   delta_step_kernel   one token: a CTA per head also computes the low-rank decay product, the head norm and the gate.
#include "stack.cuh"

namespace tbl {
namespace stack {
namespace {

using pair2 = unsigned long long;      // two packed fp32

__device__ __forceinline__ pair2 dup2(float v) { pair2 r; asm("mov.b64 %0, {%1, %1};" : "=l"(r) : "f"(v)); return r; }
__device__ __forceinline__ pair2 make2(float a, float b) { pair2 r; asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b)); return r; }
__device__ __forceinline__ void split2(pair2 v, float& a, float& b) { asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v)); }
__device__ __forceinline__ pair2 fma2(pair2 a, pair2 b, pair2 c) { pair2 d; asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c)); return d; }
__device__ __forceinline__ pair2 mul2(pair2 a, pair2 b) { pair2 d; asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b)); return d; }
__device__ __forceinline__ pair2 add2(pair2 a, pair2 b) { pair2 d; asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b)); return d; }
__device__ __forceinline__ float sum2(pair2 v) { float a, b; split2(v, a, b); return a + b; }
__device__ __forceinline__ float sum8lanes(float v) {
    v += __shfl_xor_sync(0xffffffffu, v, 1);
    v += __shfl_xor_sync(0xffffffffu, v, 2);
    v += __shfl_xor_sync(0xffffffffu, v, 4);
    return v;
}
__device__ __forceinline__ void bar_sync(int id, int n) { asm volatile("bar.sync %0, %1;" ::"r"(id), "r"(n) : "memory"); }
__device__ __forceinline__ void bar_arrive(int id, int n) { asm volatile("bar.arrive %0, %1;" ::"r"(id), "r"(n) : "memory"); }

// Four keys of one column (key index c .. c+3, clipped at dim): state <-> registers.
__device__ __forceinline__ ulonglong2 load_state4(const float* col, int c, int dim) {
    if ((dim & 3) == 0) {
        if (c >= dim) return make_ulonglong2(0, 0);
        return *reinterpret_cast<const ulonglong2*>(col + c);
    }
    const float a = c < dim ? col[c] : 0.0f, b = c + 1 < dim ? col[c + 1] : 0.0f;
    const float d = c + 2 < dim ? col[c + 2] : 0.0f, e = c + 3 < dim ? col[c + 3] : 0.0f;
    return make_ulonglong2(make2(a, b), make2(d, e));
}
__device__ __forceinline__ void store_state4(float* col, int c, int dim, ulonglong2 v) {
    if ((dim & 3) == 0) {
        if (c < dim) *reinterpret_cast<ulonglong2*>(col + c) = v;
        return;
    }
    float f[4];
    split2(v.x, f[0], f[1]);
    split2(v.y, f[2], f[3]);
#pragma unroll
    for (int i = 0; i < 4; ++i)
        if (c + i < dim) col[c + i] = f[i];
}

struct DeltaParams {
    const float* proj;       // [rows][ld]: r | k | v | g | a | w1 (raw products, biases added)
    const float* z;          // [rows][heads*dim] decay products W_w2 tanh(.) (scan kernel)
    const bf16* w2;          // [heads*dim][rank] (step kernel)
    const float* w0;         // [heads*dim]
    const float* norm;       // [heads*dim]
    float* states;           // [slots][heads][dim][dim]
    const int32_t* slots;
    float* o;                // [rows][heads*dim] raw readouts (scan kernel)
    void* out;
    int ld, heads, dim, rank, n_tok;
    float rate, key_eps, eps;
};

constexpr int kScanCols = 32;          // value columns per CTA
constexpr int kProducers = 8;          // producer warps: enough tokens in flight to cover the loads' latency
constexpr int kScanThreads = 32 * (4 + kProducers);

// The scan takes two tokens per round.  With w, u, q = a * u, k, r, v of the two tokens (0 and 1) and the state S before
// them, everything the round needs from S are four dot products per column, taken together:
//     d0 = u0.S,   e1 = (u1 w0).S,   p0 = (r0 w0).S,   p1 = (r1 w0 w1).S
// and the rest are products of the tokens with each other, the same for every column, which the producers work out:
//     d1 = e1 + (u1.k0) v0 - (u1.q0) d0
//     o0 = p0 + (r0.k0) v0 - (r0.q0) d0
//     o1 = p1 + (r1.w1 k0) v0 - (r1.w1 q0) d0 + (r1.k1) v1 - (r1.q1) d1
//     S  <- (w0 w1) S + (w1 k0) v0 - (w1 q0) d0 + k1 v1 - q1 d1
// An odd last token is followed by one that changes nothing (w = 1, the others 0).
template <int DKP>
struct ScanShape {
    static constexpr int kPairs = kProducers;                          // rounds per buffer: one per producer warp
    static constexpr int kScalars = 9 * DKP;                           // 12 products of the tokens with each other
    static constexpr int kValues = kScalars + 16;                      // v of both tokens, this CTA's columns
    static constexpr int kRecord = kValues + 2 * kScanCols;            // floats per round
    static constexpr size_t kSmem = sizeof(float) * 2 * kPairs * kRecord;
};

__device__ __forceinline__ float pick4(const float (&v)[4], int n) {
    const float a = n & 1 ? v[1] : v[0], b = n & 1 ? v[3] : v[2];
    return n & 2 ? b : a;
}
__device__ __forceinline__ float4 mul4(float4 a, float4 b) { return make_float4(a.x * b.x, a.y * b.y, a.z * b.z, a.w * b.w); }
__device__ __forceinline__ float dot4(float4 a, float4 b, float c) { return fmaf(a.x, b.x, fmaf(a.y, b.y, fmaf(a.z, b.z, fmaf(a.w, b.w, c)))); }
// (a division good to two units in the last place)
__device__ __forceinline__ float sigmoid_near(float z) { return __fdividef(1.0f, 1.0f + expf(-z)); }

template <int DKP>
__global__ void __launch_bounds__(kScanThreads) delta_scan_kernel(const DeltaParams p) {
    using Shape = ScanShape<DKP>;
    constexpr int PAIRS = Shape::kPairs, REC = Shape::kRecord;
    constexpr int G = DKP / 64;                // groups of four keys per consumer lane: 4 (l + 16 g), l = lane % 16
    constexpr int NI = (DKP + 127) / 128;      // groups of four channels per producer lane
    extern __shared__ __align__(16) float sm[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int head = blockIdx.y, seq = blockIdx.z, j0 = blockIdx.x * kScanCols;
    const int dim = p.dim, HD = p.heads * dim;
    const int chunks = (p.n_tok + 2 * PAIRS - 1) / (2 * PAIRS);
    const size_t row0 = static_cast<size_t>(seq) * p.n_tok;
    pdl_launch_dependents();
    pdl_wait();
    if (warp >= 4) {
        // ---- producers: warp w takes round w of every buffer; lane l channels 4l .. 4l + 3 (+ 128) ----
        const int pw = warp - 4;
        const bool vec = ((dim | p.ld) & 3) == 0;      // every row and head starts on 16 bytes
        auto load4 = [&](const float* base, int c, bool live) {
            float4 v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            if (!live || c >= dim) return v;
            if (vec) return *reinterpret_cast<const float4*>(base + c);
            v.x = base[c];
            if (c + 1 < dim) v.y = base[c + 1];
            if (c + 2 < dim) v.z = base[c + 2];
            if (c + 3 < dim) v.w = base[c + 3];
            return v;
        };
        float4 w0[NI], nr[2][NI], nk[2][NI], na[2][NI], nz[2][NI];
        float nv[2];
#pragma unroll
        for (int i = 0; i < NI; ++i) w0[i] = load4(p.w0 + head * dim, 4 * lane + 128 * i, true);
        auto fetch = [&](int t0) {
#pragma unroll
            for (int s = 0; s < 2; ++s) {
                const bool live = t0 + s < p.n_tok;
                const size_t at = row0 + (live ? t0 + s : 0);
                const float* row = p.proj + at * p.ld + head * dim;
                const float* zr = p.z + at * HD + head * dim;
#pragma unroll
                for (int i = 0; i < NI; ++i) {
                    const int c = 4 * lane + 128 * i;
                    nr[s][i] = load4(row, c, live);
                    nk[s][i] = load4(row + HD, c, live);
                    na[s][i] = load4(row + 4 * HD, c, live);
                    nz[s][i] = load4(zr, c, live);
                }
                nv[s] = live && j0 + lane < dim ? row[2 * HD + j0 + lane] : 0.0f;
            }
        };
        fetch(2 * pw);
        for (int ch = 0; ch < chunks; ++ch) {
            const int b = ch & 1, t0 = 2 * (ch * PAIRS + pw);
            if (ch >= 2) bar_sync(3 + b, kScanThreads);
            if (t0 < p.n_tok) {
                float4 r[2][NI], k[2][NI], u[2][NI], q[2][NI], w[2][NI];
                const float v0 = nv[0], v1 = nv[1];
                float s0 = 0.0f, s1 = 0.0f;
#pragma unroll
                for (int i = 0; i < NI; ++i) {
                    s0 = dot4(nk[0][i], nk[0][i], s0);
                    s1 = dot4(nk[1][i], nk[1][i], s1);
                }
                const float i0 = 1.0f / sqrtf(warp_sum(s0) + p.key_eps), i1 = 1.0f / sqrtf(warp_sum(s1) + p.key_eps);
                const bool second = t0 + 1 < p.n_tok;
                auto decay = [&](float z) { return expf(-p.rate * sigmoid_near(z)); };
#pragma unroll
                for (int s = 0; s < 2; ++s)
#pragma unroll
                    for (int i = 0; i < NI; ++i) {
                        const float n = s ? i1 : i0;
                        r[s][i] = nr[s][i];
                        k[s][i] = nk[s][i];
                        u[s][i] = mul4(k[s][i], make_float4(n, n, n, n));
                        q[s][i] = mul4(make_float4(sigmoid_near(na[s][i].x), sigmoid_near(na[s][i].y), sigmoid_near(na[s][i].z), sigmoid_near(na[s][i].w)), u[s][i]);
                        w[s][i] = make_float4(decay(nz[s][i].x + w0[i].x), decay(nz[s][i].y + w0[i].y), decay(nz[s][i].z + w0[i].z), decay(nz[s][i].w + w0[i].w));
                        if (s == 1 && !second) w[s][i] = make_float4(1.0f, 1.0f, 1.0f, 1.0f);
                    }
                fetch(t0 + 2 * PAIRS);
                float* rec = sm + static_cast<size_t>(b * PAIRS + pw) * REC;
                float m[8] = {};
#pragma unroll
                for (int i = 0; i < NI; ++i) {
                    const int c = 4 * lane + 128 * i;
                    const float4 k0w = mul4(w[1][i], k[0][i]), q0w = mul4(w[1][i], q[0][i]), ww = mul4(w[0][i], w[1][i]);
                    m[0] = dot4(r[0][i], k[0][i], m[0]); m[1] = dot4(r[0][i], q[0][i], m[1]);
                    m[2] = dot4(r[1][i], k0w, m[2]);     m[3] = dot4(r[1][i], q0w, m[3]);
                    m[4] = dot4(r[1][i], k[1][i], m[4]); m[5] = dot4(r[1][i], q[1][i], m[5]);
                    m[6] = dot4(u[1][i], k[0][i], m[6]); m[7] = dot4(u[1][i], q[0][i], m[7]);
                    if (c >= DKP) continue;
                    *reinterpret_cast<float4*>(rec + c) = u[0][i];
                    *reinterpret_cast<float4*>(rec + DKP + c) = mul4(u[1][i], w[0][i]);
                    *reinterpret_cast<float4*>(rec + 2 * DKP + c) = mul4(r[0][i], w[0][i]);
                    *reinterpret_cast<float4*>(rec + 3 * DKP + c) = mul4(r[1][i], ww);
                    *reinterpret_cast<float4*>(rec + 4 * DKP + c) = ww;
                    *reinterpret_cast<float4*>(rec + 5 * DKP + c) = k0w;
                    *reinterpret_cast<float4*>(rec + 6 * DKP + c) = q0w;
                    *reinterpret_cast<float4*>(rec + 7 * DKP + c) = k[1][i];
                    *reinterpret_cast<float4*>(rec + 8 * DKP + c) = q[1][i];
                }
                // the eight products over the lanes: after three exchanges a lane holds one of them, number lane / 4
                float m4[4], m2[2];
#pragma unroll
                for (int e = 0; e < 4; ++e)
                    m4[e] = (lane & 16 ? m[e + 4] : m[e]) + __shfl_xor_sync(0xffffffffu, lane & 16 ? m[e] : m[e + 4], 16);
#pragma unroll
                for (int e = 0; e < 2; ++e)
                    m2[e] = (lane & 8 ? m4[e + 2] : m4[e]) + __shfl_xor_sync(0xffffffffu, lane & 8 ? m4[e] : m4[e + 2], 8);
                float m1 = (lane & 4 ? m2[1] : m2[0]) + __shfl_xor_sync(0xffffffffu, lane & 4 ? m2[0] : m2[1], 4);
                m1 += __shfl_xor_sync(0xffffffffu, m1, 2);
                m1 += __shfl_xor_sync(0xffffffffu, m1, 1);
                // token 0: factors of v0, d0, v1, d1; token 1: the same; then those of d1
                float* sc = rec + Shape::kScalars;
                if ((lane & 3) == 0) {
                    const int e = lane >> 2;
                    sc[e < 2 ? e : e + 2] = m1;
                    if (e < 2) sc[2 + e] = 0.0f;
                }
                rec[Shape::kValues + lane] = v0;
                rec[Shape::kValues + kScanCols + lane] = v1;
            }
            __threadfence_block();
            bar_arrive(1 + b, kScanThreads);
        }
        return;
    }
    // ---- consumers: sixteen lanes share the keys of four columns ----
    const int l = lane & 15, base = lane & 16, cl = warp * 8 + (base >> 2);       // first of this lane's columns within the CTA
    float* st = p.states + (static_cast<size_t>(p.slots[seq]) * p.heads + head) * dim * dim;
    ulonglong2 S[4][G];
#pragma unroll
    for (int n = 0; n < 4; ++n)
#pragma unroll
        for (int g = 0; g < G; ++g)
            S[n][g] = j0 + cl + n < dim ? load_state4(st + static_cast<size_t>(j0 + cl + n) * dim, 4 * (l + 16 * g), dim) : make_ulonglong2(0, 0);
    // after the sums over the lanes, lane l holds dot product l / 4 of column l % 4: lanes 8 .. 15 finish the two readouts
    const int mine = l & 3, token = (l >> 2) & 1;
    const bool writes = l >= 8 && j0 + cl + mine < dim;
    float* o = p.o + (row0 + token) * HD + head * dim + j0 + cl + mine;
    for (int ch = 0; ch < chunks; ++ch) {
        const int b = ch & 1;
        bar_sync(1 + b, kScanThreads);
        const int t0 = 2 * ch * PAIRS, rounds = min(PAIRS, (p.n_tok - t0 + 1) / 2);
#pragma unroll 1
        for (int i = 0; i < rounds; ++i) {
            const float* rec = sm + static_cast<size_t>(b * PAIRS + i) * REC;
            const ulonglong2* q = reinterpret_cast<const ulonglong2*>(rec) + l;
            constexpr int V = DKP / 4;                     // 16-byte units per vector
            float x[4][4];
#pragma unroll
            for (int d = 0; d < 4; ++d) {
                ulonglong2 c[G];
#pragma unroll
                for (int g = 0; g < G; ++g) c[g] = q[d * V + 16 * g];
#pragma unroll
                for (int n = 0; n < 4; ++n) {
                    pair2 a = mul2(c[0].x, S[n][0].x), e = mul2(c[0].y, S[n][0].y);
#pragma unroll
                    for (int g = 1; g < G; ++g) { a = fma2(c[g].x, S[n][g].x, a); e = fma2(c[g].y, S[n][g].y, e); }
                    x[d][n] = sum2(add2(a, e));
                }
            }
            const float4 va = *reinterpret_cast<const float4*>(rec + Shape::kValues + cl), vb = *reinterpret_cast<const float4*>(rec + Shape::kValues + kScanCols + cl);
            const float4 f = *reinterpret_cast<const float4*>(rec + Shape::kScalars + 4 * token);
            const float2 fd = *reinterpret_cast<const float2*>(rec + Shape::kScalars + 8);
            float y[2][4], z[4], h[2], r;
#pragma unroll
            for (int d = 0; d < 2; ++d)
#pragma unroll
                for (int n = 0; n < 4; ++n) y[d][n] = (l & 8 ? x[d + 2][n] : x[d][n]) + __shfl_xor_sync(0xffffffffu, l & 8 ? x[d][n] : x[d + 2][n], 8);
#pragma unroll
            for (int n = 0; n < 4; ++n) z[n] = (l & 4 ? y[1][n] : y[0][n]) + __shfl_xor_sync(0xffffffffu, l & 4 ? y[0][n] : y[1][n], 4);
#pragma unroll
            for (int n = 0; n < 2; ++n) h[n] = (l & 2 ? z[n + 2] : z[n]) + __shfl_xor_sync(0xffffffffu, l & 2 ? z[n] : z[n + 2], 2);
            r = (l & 1 ? h[1] : h[0]) + __shfl_xor_sync(0xffffffffu, l & 1 ? h[0] : h[1], 1);
            float d0[4], d1[4];
            const float v0[4] = {va.x, va.y, va.z, va.w}, v1[4] = {vb.x, vb.y, vb.z, vb.w};
#pragma unroll
            for (int n = 0; n < 4; ++n) {
                d0[n] = __shfl_sync(0xffffffffu, r, base + n);
                d1[n] = __shfl_sync(0xffffffffu, r, base + 4 + n);
            }
#pragma unroll
            for (int n = 0; n < 4; ++n) d1[n] = fmaf(fd.x, v0[n], fmaf(-fd.y, d0[n], d1[n]));
            pair2 p0[4], p1[4], m0[4], m1[4];
#pragma unroll
            for (int n = 0; n < 4; ++n) { p0[n] = dup2(v0[n]); p1[n] = dup2(v1[n]); m0[n] = dup2(-d0[n]); m1[n] = dup2(-d1[n]); }
#pragma unroll
            for (int g = 0; g < G; ++g) {
                const ulonglong2 w = q[4 * V + 16 * g], k0 = q[5 * V + 16 * g], q0 = q[6 * V + 16 * g], k1 = q[7 * V + 16 * g], q1 = q[8 * V + 16 * g];
#pragma unroll
                for (int n = 0; n < 4; ++n) {
                    S[n][g].x = fma2(q1.x, m1[n], fma2(k1.x, p1[n], fma2(q0.x, m0[n], fma2(k0.x, p0[n], mul2(w.x, S[n][g].x)))));
                    S[n][g].y = fma2(q1.y, m1[n], fma2(k1.y, p1[n], fma2(q0.y, m0[n], fma2(k0.y, p0[n], mul2(w.y, S[n][g].y)))));
                }
            }
            const float out = fmaf(f.x, pick4(v0, mine), fmaf(-f.y, pick4(d0, mine), fmaf(f.z, pick4(v1, mine), fmaf(-f.w, pick4(d1, mine), r))));
            if (writes && t0 + 2 * i + token < p.n_tok) o[static_cast<size_t>(t0 + 2 * i) * HD] = out;
        }
        if (ch + 2 < chunks) bar_arrive(3 + b, kScanThreads);
    }
#pragma unroll
    for (int n = 0; n < 4; ++n)
#pragma unroll
        for (int g = 0; g < G; ++g)
            if (j0 + cl + n < dim) store_state4(st + static_cast<size_t>(j0 + cl + n) * dim, 4 * (l + 16 * g), dim, S[n][g]);
}

// tanh of the low-rank decay projection, in the precision's type, for the GEMM with W_w2
template <typename T>
__global__ void __launch_bounds__(256) delta_tanh_kernel(const float* __restrict__ proj, int ld, int offset, int rows, int rank,
                                                         int ldt, T* __restrict__ out) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t i = static_cast<size_t>(blockIdx.x) * 256 + threadIdx.x;
    const size_t row = i / rank;
    const int c = static_cast<int>(i - row * rank);
    if (row < static_cast<size_t>(rows)) out[row * ldt + c] = from_f<T>(tanhf(proj[row * ld + offset + c]));
}

// head norm, weight and output gate of the scan's readouts: one warp per (row, head)
template <typename T>
__global__ void __launch_bounds__(256) delta_out_kernel(const DeltaParams p, int rows) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t unit = static_cast<size_t>(blockIdx.x) * 8 + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31, dim = p.dim, HD = p.heads * dim;
    if (unit >= static_cast<size_t>(rows) * p.heads) return;
    const size_t row = unit / p.heads;
    const int head = static_cast<int>(unit - row * p.heads);
    const float* o = p.o + row * HD + head * dim;
    const float* g = p.proj + row * p.ld + 3 * HD + head * dim;
    T* out = static_cast<T*>(p.out) + row * HD + head * dim;
    float ov[TBL_MAX_DELTA_DIM / 32], gv[TBL_MAX_DELTA_DIM / 32], ss = 0.0f;
#pragma unroll
    for (int i = 0; i < TBL_MAX_DELTA_DIM / 32; ++i) {
        const int c = lane + 32 * i;
        ov[i] = c < dim ? o[c] : 0.0f;
        gv[i] = c < dim ? g[c] : 0.0f;
        ss = fmaf(ov[i], ov[i], ss);
    }
    const float inv = 1.0f / sqrtf(warp_sum(ss) / static_cast<float>(dim) + p.eps);
#pragma unroll
    for (int i = 0; i < TBL_MAX_DELTA_DIM / 32; ++i) {
        const int c = lane + 32 * i;
        if (c < dim) out[c] = from_f<T>(ov[i] * inv * __ldg(p.norm + head * dim + c) * sigmoid_f(gv[i]));
    }
}

// ---- one token ------------------------------------------------------------------------------------------------------
// THREADS / 8 column groups; a thread's columns are its group + i * THREADS / 8, taken NCP at a time.
template <typename T, int DKP, int THREADS, int NCP, bool FUSED>
__global__ void __launch_bounds__(THREADS, DKP == 128 ? 2 : 1) delta_step_kernel(const DeltaParams p) {
    constexpr int G = DKP / 32, GROUPS = THREADS / 8, PASSES = DKP / (GROUPS * NCP);
    static_assert(PASSES >= 1 && PASSES * GROUPS * NCP == DKP, "columns of a head");
    __shared__ __align__(16) float su[DKP], sw[DKP], sau[DKP], sk[DKP], sr[DKP], sv[DKP], so[DKP], part[FUSED ? THREADS : 1];
    extern __shared__ float st_tanh[];         // [rank]
    const int tid = threadIdx.x, lane = tid & 31;
    const int head = blockIdx.x, row = blockIdx.y;
    const int dim = p.dim, HD = p.heads * dim;
    pdl_launch_dependents();
    float* st = p.states + (static_cast<size_t>(p.slots[row]) * p.heads + head) * dim * dim;
    for (int e = tid * 32; e < dim * dim; e += THREADS * 32) asm volatile("prefetch.global.L2 [%0];" ::"l"(st + e));
    pdl_wait();
    const float* pr = p.proj + static_cast<size_t>(row) * p.ld;
    const int l8 = tid & 7, group = tid >> 3;
    ulonglong2 S[NCP][G];
    auto load_pass = [&](int ps) {
#pragma unroll
        for (int n = 0; n < NCP; ++n) {
            const int j = (ps * NCP + n) * GROUPS + group;
#pragma unroll
            for (int g = 0; g < G; ++g)
                S[n][g] = j < dim ? load_state4(st + static_cast<size_t>(j) * dim, 4 * (l8 + 8 * g), dim) : make_ulonglong2(0, 0);
        }
    };
    // everything that depends on this step's projections is requested first, then the state
    const int hc = head * dim + tid;
    const bool ch = tid < dim;
    const float k_in = ch ? pr[HD + hc] : 0.0f, r_in = ch ? pr[hc] : 0.0f, v_in = ch ? pr[2 * HD + hc] : 0.0f;
    const float g_in = ch ? pr[3 * HD + hc] : 0.0f, a_in = ch ? pr[4 * HD + hc] : 0.0f;
    float z_in = !FUSED && ch ? p.z[static_cast<size_t>(row) * HD + hc] : 0.0f;
    float kn[DKP / 32];
#pragma unroll
    for (int i = 0; i < DKP / 32; ++i) kn[i] = lane + 32 * i < dim ? pr[HD + head * dim + lane + 32 * i] : 0.0f;
    load_pass(0);
    if constexpr (FUSED) {
        for (int e = tid; e < p.rank; e += THREADS) st_tanh[e] = tanhf(pr[5 * HD + e]);
        __syncthreads();
        // decay products: THREADS / DKP threads per channel
        constexpr int TPC = THREADS / DKP;
        const int c = tid / TPC, sub = tid % TPC;
        float z = 0.0f;
        if (c < dim) {
            const bf16* w2 = p.w2 + static_cast<size_t>(head * dim + c) * p.rank;
            if ((p.rank & 7) == 0) {
#pragma unroll 4
                for (int e = sub * 8; e < p.rank; e += TPC * 8) {
                    const uint4 w = __ldg(reinterpret_cast<const uint4*>(w2 + e));
                    z = fmaf(bf_lo(w.x), st_tanh[e], z); z = fmaf(bf_hi(w.x), st_tanh[e + 1], z);
                    z = fmaf(bf_lo(w.y), st_tanh[e + 2], z); z = fmaf(bf_hi(w.y), st_tanh[e + 3], z);
                    z = fmaf(bf_lo(w.z), st_tanh[e + 4], z); z = fmaf(bf_hi(w.z), st_tanh[e + 5], z);
                    z = fmaf(bf_lo(w.w), st_tanh[e + 6], z); z = fmaf(bf_hi(w.w), st_tanh[e + 7], z);
                }
            } else {
                for (int e = sub; e < p.rank; e += TPC) z = fmaf(to_f(w2[e]), st_tanh[e], z);
            }
        }
        part[tid] = z;
        __syncthreads();
        if (ch) {
#pragma unroll
            for (int s = 0; s < TPC; ++s) z_in += part[tid * TPC + s];
        }
    }
    float ss = 0.0f;                            // every warp takes the key's norm for itself
#pragma unroll
    for (int i = 0; i < DKP / 32; ++i) ss = fmaf(kn[i], kn[i], ss);
    const float inv_key = 1.0f / sqrtf(warp_sum(ss) + p.key_eps);
    if (tid < DKP) {
        const float u = k_in * inv_key;
        su[tid] = u;
        sk[tid] = k_in;
        sr[tid] = r_in;
        sv[tid] = v_in;
        sw[tid] = ch ? expf(-p.rate * sigmoid_f(z_in + __ldg(p.w0 + hc))) : 0.0f;
        sau[tid] = sigmoid_f(a_in) * u;
    }
    __syncthreads();
    const ulonglong2 *qu = reinterpret_cast<const ulonglong2*>(su) + l8, *qw = reinterpret_cast<const ulonglong2*>(sw) + l8,
                     *qa = reinterpret_cast<const ulonglong2*>(sau) + l8, *qk = reinterpret_cast<const ulonglong2*>(sk) + l8,
                     *qr = reinterpret_cast<const ulonglong2*>(sr) + l8;
#pragma unroll 1
    for (int ps = 0; ps < PASSES; ++ps) {
        if (ps > 0) load_pass(ps);
        pair2 m[NCP], vv[NCP];
#pragma unroll
        for (int n = 0; n < NCP; ++n) {
            pair2 d = 0, e = 0;
#pragma unroll
            for (int g = 0; g < G; ++g) { d = fma2(qu[8 * g].x, S[n][g].x, d); e = fma2(qu[8 * g].y, S[n][g].y, e); }
            m[n] = dup2(-sum8lanes(sum2(add2(d, e))));
            vv[n] = dup2(sv[(ps * NCP + n) * GROUPS + group]);
        }
#pragma unroll
        for (int n = 0; n < NCP; ++n) {
            const int j = (ps * NCP + n) * GROUPS + group;
            pair2 o = 0, f = 0;
#pragma unroll
            for (int g = 0; g < G; ++g) {
                S[n][g].x = fma2(qw[8 * g].x, S[n][g].x, fma2(qa[8 * g].x, m[n], mul2(qk[8 * g].x, vv[n])));
                S[n][g].y = fma2(qw[8 * g].y, S[n][g].y, fma2(qa[8 * g].y, m[n], mul2(qk[8 * g].y, vv[n])));
                o = fma2(qr[8 * g].x, S[n][g].x, o);
                f = fma2(qr[8 * g].y, S[n][g].y, f);
                if (j < dim) store_state4(st + static_cast<size_t>(j) * dim, 4 * (l8 + 8 * g), dim, S[n][g]);
            }
            const float r = sum8lanes(sum2(add2(o, f)));
            if (l8 == 0) so[j] = r;
        }
    }
    __syncthreads();
    float sq = 0.0f;
#pragma unroll
    for (int i = 0; i < DKP / 32; ++i) { const float v = so[lane + 32 * i]; sq = fmaf(v, v, sq); }   // zero past dim
    const float inv = 1.0f / sqrtf(warp_sum(sq) / static_cast<float>(dim) + p.eps);
    if (ch) static_cast<T*>(p.out)[static_cast<size_t>(row) * HD + hc] = from_f<T>(so[tid] * inv * __ldg(p.norm + hc) * sigmoid_f(g_in));
}

// From this many rows on W_w2 is one product over all of them instead of a part of every head's CTA.
constexpr int kStepFusedRows = 4;

// z = W_w2 tanh(low-rank part), fp32 [rows][heads*dim]
template <typename T>
int decay_products(const tbl_delta_mixer& m, const DeltaParams& p, int precision, int rows, T* th, float* z, cudaStream_t st) {
    const int HD = p.heads * p.dim, ldt = static_cast<int>(round_up(p.rank, 8));
    if (launch_dependent(delta_tanh_kernel<T>, dim3(ceil_div(static_cast<long long>(rows) * p.rank, 256)), dim3(256), 0, st, p.proj, p.ld, 5 * HD,
                         rows, p.rank, ldt, th) != cudaSuccess)
        return TBL_ERR_CUDA;
    DenseCall c{};
    c.x = th; c.w = static_cast<const bf16*>(m.decay_up.weight); c.ldx = ldt; c.M = rows; c.K = p.rank; c.N = HD;
    c.out_f32 = z; c.ldo = HD;
    return launch_dense(precision, kDenseAuto, c, st);
}

template <typename T, int DKP, int THREADS, int NCP>
cudaError_t launch_step_d(const DeltaParams& p, dim3 grid, cudaStream_t st) {
    return p.z ? launch_dependent(delta_step_kernel<T, DKP, THREADS, NCP, false>, grid, dim3(THREADS), 0, st, p)
               : launch_dependent(delta_step_kernel<T, DKP, THREADS, NCP, true>, grid, dim3(THREADS), sizeof(float) * p.rank, st, p);
}

struct Workspace {
    float *z, *o;
    void* th;
    size_t bytes;
};
Workspace carve(const tbl_delta_mixer& m, int precision, size_t rows, void* base) {
    Workspace w{};
    const size_t HD = static_cast<size_t>(m.heads) * m.dim, e = precision == TBL_BF16 ? 2 : 4;
    uint8_t* p = static_cast<uint8_t*>(base);
    auto take = [&](size_t bytes) { uint8_t* r = p + w.bytes; w.bytes += round_up(bytes, 256); return r; };
    w.z = reinterpret_cast<float*>(take(sizeof(float) * rows * HD));
    w.o = reinterpret_cast<float*>(take(sizeof(float) * rows * HD));
    w.th = take(e * rows * round_up(m.rank, 8));
    return w;
}

template <typename T>
int launch_step(const tbl_delta_mixer& m, DeltaParams p, int precision, int n_seq, void* ws, cudaStream_t st) {
    const dim3 grid(p.heads, n_seq);
    if (n_seq > 65535 || p.rank > 8192) return TBL_ERR_SHAPE;
    if (n_seq >= kStepFusedRows) {
        const Workspace w = carve(m, precision, n_seq, ws);
        const int rc = decay_products<T>(m, p, precision, n_seq, static_cast<T*>(w.th), w.z, st);
        if (rc != TBL_OK) return rc;
        p.z = w.z;
    }
    cudaError_t e;
    if (p.dim <= 32) e = launch_step_d<T, 32, 256, 1>(p, grid, st);
    else if (p.dim <= 64) e = launch_step_d<T, 64, 256, 2>(p, grid, st);
    else if (p.dim <= 128) e = launch_step_d<T, 128, 256, 4>(p, grid, st);
    else e = launch_step_d<T, 256, 512, 1>(p, grid, st);
    return e == cudaSuccess ? TBL_OK : TBL_ERR_CUDA;
}

template <int DKP>
int launch_scan_d(const DeltaParams& p, int n_seq, cudaStream_t st) {
    static bool done[64] = {};
    if (allow_smem(delta_scan_kernel<DKP>, ScanShape<DKP>::kSmem, done) != cudaSuccess) return TBL_ERR_CUDA;
    const dim3 grid(ceil_div(p.dim, kScanCols), p.heads, n_seq);
    if (p.heads > 65535 || n_seq > 65535) return TBL_ERR_SHAPE;
    return launch_dependent(delta_scan_kernel<DKP>, grid, dim3(kScanThreads), ScanShape<DKP>::kSmem, st, p) == cudaSuccess ? TBL_OK
                                                                                                                      : TBL_ERR_CUDA;
}

template <typename T>
int launch_scan(const tbl_delta_mixer& m, DeltaParams p, int precision, int n_seq, void* ws, cudaStream_t st) {
    const int rows = n_seq * p.n_tok;
    const Workspace w = carve(m, precision, rows, ws);
    p.o = w.o;
    int rc = decay_products<T>(m, p, precision, rows, static_cast<T*>(w.th), w.z, st);
    if (rc != TBL_OK) return rc;
    p.z = w.z;
    if (p.dim <= 64) rc = launch_scan_d<64>(p, n_seq, st);
    else if (p.dim <= 128) rc = launch_scan_d<128>(p, n_seq, st);
    else rc = launch_scan_d<256>(p, n_seq, st);
    if (rc != TBL_OK) return rc;
    const cudaError_t e = launch_dependent(delta_out_kernel<T>, dim3(ceil_div(static_cast<long long>(rows) * p.heads, 8)), dim3(256), 0, st, p, rows);
    return e == cudaSuccess ? TBL_OK : TBL_ERR_CUDA;
}

}  // namespace

int check_delta(const tbl_delta_mixer& m, int width) {
    if (m.heads <= 0 || m.dim <= 0 || m.dim > TBL_MAX_DELTA_DIM || m.rank <= 0) return TBL_ERR_SHAPE;
    const int HD = m.heads * m.dim;
    if (m.in.inputs != width || m.in.outputs != 5 * HD + m.rank || m.decay_up.inputs != m.rank || m.decay_up.outputs != HD ||
        m.out.inputs != HD || m.out.outputs != width)
        return TBL_ERR_SHAPE;
    if (!m.in.weight || !m.in.bias || !m.decay_up.weight || !m.decay_up.bias || !m.out.weight || !m.norm) return TBL_ERR_INVALID_ARG;
    return TBL_OK;
}

size_t delta_workspace(const tbl_delta_mixer& m, int precision, int rows) { return carve(m, precision, rows, nullptr).bytes; }

int launch_delta(const tbl_delta_mixer& m, int precision, int route, float eps, const float* proj, float* states,
                 const int32_t* slots, int n_seq, int n_tok, void* out, void* ws, cudaStream_t st) {
    DeltaParams p{};
    p.proj = proj; p.w2 = static_cast<const bf16*>(m.decay_up.weight); p.w0 = m.decay_up.bias; p.norm = m.norm;
    p.states = states; p.slots = slots; p.out = out; p.ld = m.in.outputs; p.heads = m.heads; p.dim = m.dim; p.rank = m.rank;
    p.n_tok = n_tok; p.rate = m.decay_rate; p.key_eps = m.key_eps; p.eps = eps;
    if (route == 0) route = n_tok == 1 ? 2 : 1;
    if (route == 2) {
        if (n_tok != 1) return TBL_ERR_SHAPE;
        return precision == TBL_BF16 ? launch_step<bf16>(m, p, precision, n_seq, ws, st) : launch_step<float>(m, p, precision, n_seq, ws, st);
    }
    if (route != 1) return TBL_ERR_INVALID_ARG;
    return precision == TBL_BF16 ? launch_scan<bf16>(m, p, precision, n_seq, ws, st) : launch_scan<float>(m, p, precision, n_seq, ws, st);
}

}  // namespace stack
}  // namespace tbl

using namespace tbl;
using namespace tbl::stack;

extern "C" {

size_t tbl_delta_workspace_bytes(const tbl_delta_mixer* mixer, int precision, int rows) {
    return mixer && rows > 0 ? delta_workspace(*mixer, precision, rows) : 0;
}

int tbl_delta_forward(const tbl_delta_mixer* mixer, int precision, int route, float eps, const float* proj_dev, float* states_dev,
                      const int32_t* slots_dev, int n_seq, int n_tok, void* out_dev, void* workspace_dev, size_t workspace_bytes,
                      void* stream) {
    if (!mixer || !proj_dev || !states_dev || !slots_dev || !out_dev || n_seq <= 0 || n_tok <= 0 ||
        (precision != TBL_F32 && precision != TBL_BF16))
        return TBL_ERR_INVALID_ARG;
    const int rc = check_delta(*mixer, mixer->in.inputs);
    if (rc != TBL_OK) return rc;
    if (!workspace_dev || workspace_bytes < delta_workspace(*mixer, precision, n_seq * n_tok)) return TBL_ERR_WORKSPACE;
    if ((reinterpret_cast<uintptr_t>(workspace_dev) & 255) || (reinterpret_cast<uintptr_t>(states_dev) & 15)) return TBL_ERR_ALIGNMENT;
    return launch_delta(*mixer, precision, route, eps, proj_dev, states_dev, slots_dev, n_seq, n_tok, out_dev, workspace_dev,
                        static_cast<cudaStream_t>(stream));
}

}  // extern "C"
