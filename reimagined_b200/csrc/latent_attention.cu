// Latent attention: keys and values are linear images of a cached latent, plus one rotated key part shared by the
// heads, so a token costs kv_rank + rot_dim cached numbers whatever the head count.
//
//   latent_prep_kernel     norms of the query latent and of the cached latent, rotation of the shared key part, append
//   latent_absorb_kernel   (fp32 and odd sizes) query side of W_uk: q' = W_uk^T q per head (and the rotation of the query's rotated part), so
//                          that scores are dot products with the cache itself
//   latent_simt_kernel     attention over the cache, any sizes, fp32 arithmetic; split over the context
//   latent_value_kernel    merges the splits, applies W_uv per head and the output gate
// Scores, softmax weights and their sums are fp32 throughout.
#include "latent.cuh"

namespace tbl {
namespace stack {
namespace {

// One CTA per row of the step; a thread keeps its numbers in registers between the sum of squares and the stores.
constexpr int kPrepThreads = 256, kPrepQ = 8, kPrepC = TBL_MAX_LATENT / kPrepThreads;

template <typename T>
__global__ void __launch_bounds__(kPrepThreads) latent_prep_kernel(const LatentParams p) {
    __shared__ float red[2][kPrepThreads / 32];
    pdl_launch_dependents();
    pdl_wait();
    const int row = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int slot = p.slots[row / p.n_tok];
    const int pos = p.positions[slot] + row % p.n_tok;
    const float* pr = p.proj + static_cast<size_t>(row) * p.ld;
    const float* kv = pr + p.q_rank;
    float q[kPrepQ], c[kPrepC], sq = 0.0f, sc = 0.0f;
#pragma unroll
    for (int i = 0; i < kPrepQ; ++i) { const int e = tid + i * kPrepThreads; q[i] = e < p.q_rank ? pr[e] : 0.0f; }
#pragma unroll
    for (int i = 0; i < kPrepC; ++i) { const int e = tid + i * kPrepThreads; c[i] = e < p.R ? kv[e] : 0.0f; }
    const bool room = pos >= 0 && pos < p.capacity && pos < p.rope_positions;
    const int half = p.rd / 2, at = room ? pos : 0;
    float u = 0.0f, v = 0.0f, cv = 0.0f, sv = 0.0f;
    if (tid < half) {                                      // rd <= TBL_MAX_LATENT: one pair per thread for up to 512 dimensions
        u = kv[p.R + tid]; v = kv[p.R + tid + half];
        cv = __ldg(p.rope_cos + static_cast<size_t>(at) * half + tid); sv = __ldg(p.rope_sin + static_cast<size_t>(at) * half + tid);
    }
#pragma unroll
    for (int i = 0; i < kPrepQ; ++i) sq = fmaf(q[i], q[i], sq);
    for (int e = tid + kPrepQ * kPrepThreads; e < p.q_rank; e += kPrepThreads) sq = fmaf(pr[e], pr[e], sq);
#pragma unroll
    for (int i = 0; i < kPrepC; ++i) sc = fmaf(c[i], c[i], sc);
    sq = warp_sum(sq);
    sc = warp_sum(sc);
    if (lane == 0) { red[0][warp] = sq; red[1][warp] = sc; }
    __syncthreads();
    sq = sc = 0.0f;
#pragma unroll
    for (int w = 0; w < kPrepThreads / 32; ++w) { sq += red[0][w]; sc += red[1][w]; }
    const float iq = 1.0f / sqrtf(sq / static_cast<float>(p.q_rank) + p.eps);
    const float ic = 1.0f / sqrtf(sc / static_cast<float>(p.R) + p.eps);
    T* cq = static_cast<T*>(p.cq) + static_cast<size_t>(row) * p.ldq;
#pragma unroll
    for (int i = 0; i < kPrepQ; ++i) { const int e = tid + i * kPrepThreads; if (e < p.q_rank) cq[e] = from_f<T>(q[i] * iq * __ldg(p.q_norm + e)); }
    for (int e = tid + kPrepQ * kPrepThreads; e < p.q_rank; e += kPrepThreads) cq[e] = from_f<T>(pr[e] * iq * __ldg(p.q_norm + e));
    if (!room) {
        if (tid == 0) atomicOr(p.status, TBL_DEV_CACHE_FULL);
        return;
    }
    T* out = static_cast<T*>(p.cache) + (static_cast<size_t>(slot) * p.capacity + pos) * p.cw;
#pragma unroll
    for (int i = 0; i < kPrepC; ++i) { const int e = tid + i * kPrepThreads; if (e < p.R) out[e] = from_f<T>(c[i] * ic * __ldg(p.kv_norm + e)); }
    if (tid < half) {
        out[p.R + tid] = from_f<T>(u * cv - v * sv);
        out[p.R + half + tid] = from_f<T>(v * cv + u * sv);
    }
    for (int i = tid + kPrepThreads; i < half; i += kPrepThreads) {
        const float a = kv[p.R + i], b = kv[p.R + i + half];
        const float ci = __ldg(p.rope_cos + static_cast<size_t>(pos) * half + i), si = __ldg(p.rope_sin + static_cast<size_t>(pos) * half + i);
        out[p.R + i] = from_f<T>(a * ci - b * si);
        out[p.R + half + i] = from_f<T>(b * ci + a * si);
    }
}

// One CTA per (row, head): q' [R] = sum_d q[d] W_uk[head, d, :], then the rotated part of q.
template <typename T>
__global__ void __launch_bounds__(128) latent_absorb_kernel(const LatentParams p) {
    extern __shared__ float q[];                  // [d + rd]
    pdl_launch_dependents();
    const int row = blockIdx.x, head = blockIdx.y, tid = threadIdx.x, n = p.d + p.rd;
    pdl_wait();
    const int slot = p.slots[row / p.n_tok];
    const int pos = min(max(p.positions[slot] + row % p.n_tok, 0), p.rope_positions - 1);
    const float* qr = p.q + (static_cast<size_t>(row) * p.H + head) * n;
    for (int e = tid; e < n; e += 128) q[e] = qr[e];
    __syncthreads();
    T* out = static_cast<T*>(p.qa) + (static_cast<size_t>(row) * p.H + head) * p.cw;
    const bf16* w = p.uk + static_cast<size_t>(head) * p.d * p.R;
    if ((p.R & 1) == 0) {
        for (int e = 2 * tid; e < p.R; e += 256) {
            float a = 0.0f, b = 0.0f;
#pragma unroll 16
            for (int k = 0; k < p.d; ++k) {
                const uint32_t v = __ldg(reinterpret_cast<const uint32_t*>(w + static_cast<size_t>(k) * p.R + e));
                a = fmaf(q[k], bf_lo(v), a);
                b = fmaf(q[k], bf_hi(v), b);
            }
            out[e] = from_f<T>(a);
            out[e + 1] = from_f<T>(b);
        }
    } else {
        for (int e = tid; e < p.R; e += 128) {
            float a = 0.0f;
            for (int k = 0; k < p.d; ++k) a = fmaf(q[k], to_f(w[static_cast<size_t>(k) * p.R + e]), a);
            out[e] = from_f<T>(a);
        }
    }
    const int half = p.rd / 2;
    for (int i = tid; i < half; i += 128) {
        const float cv = __ldg(p.rope_cos + static_cast<size_t>(pos) * half + i), sv = __ldg(p.rope_sin + static_cast<size_t>(pos) * half + i);
        const float u = q[p.d + i], v = q[p.d + half + i];
        out[p.R + i] = from_f<T>(u * cv - v * sv);
        out[p.R + half + i] = from_f<T>(v * cv + u * sv);
    }
    for (int e = p.R + p.rd + tid; e < p.cw; e += 128) out[e] = from_f<T>(0.0f);
}

// One CTA of four warps per (row, head, split); a warp takes every fourth token pair of the split, lanes share the
// numbers of a cached token: element lane + 32 i.
constexpr int kSimtWarps = 4;

template <typename T, int NI>
__global__ void __launch_bounds__(32 * kSimtWarps) latent_simt_kernel(const LatentParams p) {
    __shared__ float acc_s[kSimtWarps][NI * 32], m_s[kSimtWarps], l_s[kSimtWarps];
    pdl_launch_dependents();
    const int row = blockIdx.x, head = blockIdx.y, split = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    pdl_wait();
    const int slot = p.slots[row / p.n_tok];
    const int n = min(p.positions[slot] + row % p.n_tok + 1, p.capacity);       // visible tokens
    const int per = (n + p.splits - 1) / p.splits;
    const int t0 = split * per, t1 = min(n, t0 + per);
    const int CW = p.R + p.rd;
    const T* qa = static_cast<const T*>(p.qa) + (static_cast<size_t>(row) * p.H + head) * p.cw;
    const T* cache = static_cast<const T*>(p.cache) + static_cast<size_t>(slot) * p.capacity * p.cw;
    float q[NI], acc[NI];
#pragma unroll
    for (int i = 0; i < NI; ++i) { q[i] = lane + 32 * i < CW ? to_f(qa[lane + 32 * i]) : 0.0f; acc[i] = 0.0f; }
    float m = -INFINITY, l = 0.0f;
    for (int t = t0 + 2 * warp; t < t1; t += 2 * kSimtWarps) {
        const bool two = t + 1 < t1;
        float c0[NI], c1[NI], s0 = 0.0f, s1 = 0.0f;
        const T* r0 = cache + static_cast<size_t>(t) * p.cw;
        const T* r1 = two ? r0 + p.cw : r0;
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const bool ok = lane + 32 * i < CW;
            c0[i] = ok ? to_f(r0[lane + 32 * i]) : 0.0f;
            c1[i] = ok ? to_f(r1[lane + 32 * i]) : 0.0f;
        }
#pragma unroll
        for (int i = 0; i < NI; ++i) { s0 = fmaf(q[i], c0[i], s0); s1 = fmaf(q[i], c1[i], s1); }
        s0 = warp_sum(s0) * p.scale;
        s1 = two ? warp_sum(s1) * p.scale : -INFINITY;
        const float mn = fmaxf(m, fmaxf(s0, s1));
        const float a = expf(m - mn), p0 = expf(s0 - mn), p1 = expf(s1 - mn);
        l = fmaf(l, a, p0 + p1);
        m = mn;
#pragma unroll
        for (int i = 0; i < NI; ++i) acc[i] = fmaf(acc[i], a, fmaf(p0, c0[i], p1 * c1[i]));
    }
#pragma unroll
    for (int i = 0; i < NI; ++i) acc_s[warp][lane + 32 * i] = acc[i];
    if (lane == 0) { m_s[warp] = m; l_s[warp] = l; }
    __syncthreads();
    float mt = m_s[0];
#pragma unroll
    for (int w = 1; w < kSimtWarps; ++w) mt = fmaxf(mt, m_s[w]);
    float f[kSimtWarps], lt = 0.0f;
#pragma unroll
    for (int w = 0; w < kSimtWarps; ++w) { f[w] = m_s[w] == -INFINITY ? 0.0f : expf(m_s[w] - mt); lt = fmaf(l_s[w], f[w], lt); }
    const size_t unit = (static_cast<size_t>(row) * p.H + head) * p.splits + split;
    for (int e = tid; e < p.R; e += 32 * kSimtWarps) {
        float v = 0.0f;
#pragma unroll
        for (int w = 0; w < kSimtWarps; ++w) v = fmaf(acc_s[w][e], f[w], v);
        p.part_o[unit * p.R + e] = v;
    }
    if (tid == 0) { p.part_m[unit] = mt; p.part_l[unit] = lt; }
}

// One CTA per (row, head): merge, W_uv, gate.
template <typename T>
__global__ void __launch_bounds__(256) latent_value_kernel(const LatentParams p) {
    extern __shared__ float sm[];                // [R] latent | [splits] factors
    float* lat = sm;
    float* fac = sm + p.R;
    __shared__ float total_s;
    pdl_launch_dependents();
    const int row = blockIdx.x, head = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    pdl_wait();
    const size_t unit = (static_cast<size_t>(row) * p.H + head) * p.splits;
    if (warp == 0) {
        float m = -INFINITY, l = 0.0f;
        for (int s = lane; s < p.splits; s += 32) m = fmaxf(m, p.part_m[unit + s]);
        m = warp_max(m);
        for (int s = lane; s < p.splits; s += 32) {
            const float ms = p.part_m[unit + s], f = ms == -INFINITY ? 0.0f : expf(ms - m);
            fac[s] = f;
            l = fmaf(p.part_l[unit + s], f, l);
        }
        l = warp_sum(l);
        if (lane == 0) total_s = 1.0f / l;
    }
    __syncthreads();
    for (int e = tid; e < p.R; e += 256) {
        float v = 0.0f;
#pragma unroll 4
        for (int s = 0; s < p.splits; ++s) v = fmaf(p.part_o[(unit + s) * p.R + e], fac[s], v);
        lat[e] = v * total_s;
    }
    __syncthreads();
    const float* g = p.proj + static_cast<size_t>(row) * p.ld + p.q_rank + p.R + p.rd + head * p.vd;
    T* out = static_cast<T*>(p.out) + static_cast<size_t>(row) * p.H * p.vd + head * p.vd;
    for (int v = warp; v < p.vd; v += 8) {
        const bf16* w = p.uv + static_cast<size_t>(head * p.vd + v) * p.R;
        float a = 0.0f;
        if ((p.R & 7) == 0) {
            for (int e = lane * 8; e < p.R; e += 256) {
                const uint4 x = __ldg(reinterpret_cast<const uint4*>(w + e));
                const float4 s = *reinterpret_cast<const float4*>(lat + e), t = *reinterpret_cast<const float4*>(lat + e + 4);
                a = fmaf(bf_lo(x.x), s.x, a); a = fmaf(bf_hi(x.x), s.y, a); a = fmaf(bf_lo(x.y), s.z, a); a = fmaf(bf_hi(x.y), s.w, a);
                a = fmaf(bf_lo(x.z), t.x, a); a = fmaf(bf_hi(x.z), t.y, a); a = fmaf(bf_lo(x.w), t.z, a); a = fmaf(bf_hi(x.w), t.w, a);
            }
        } else {
            for (int e = lane; e < p.R; e += 32) a = fmaf(to_f(w[e]), lat[e], a);
        }
        a = warp_sum(a);
        if (lane == 0) out[v] = from_f<T>(a * sigmoid_f(g[v]));
    }
}

template <typename T>
int launch_simt(const LatentParams& p, int rows, cudaStream_t st) {
    const dim3 grid(rows, p.H, p.splits);
    const int CW = p.R + p.rd;
    cudaError_t e;
    if (CW <= 128) e = launch_dependent(latent_simt_kernel<T, 4>, grid, dim3(32 * kSimtWarps), 0, st, p);
    else if (CW <= 320) e = launch_dependent(latent_simt_kernel<T, 10>, grid, dim3(32 * kSimtWarps), 0, st, p);
    else if (CW <= 576) e = launch_dependent(latent_simt_kernel<T, 18>, grid, dim3(32 * kSimtWarps), 0, st, p);
    else e = launch_dependent(latent_simt_kernel<T, 32>, grid, dim3(32 * kSimtWarps), 0, st, p);
    return e == cudaSuccess ? TBL_OK : TBL_ERR_CUDA;
}

enum Route { kAuto = 0, kCacheSimt = 1, kCacheTensor = 2, kExpanded = 3 };
// From this many new tokens of a sequence on, expanding keys and values of the whole context costs less than running
// the attention in the latent space.
constexpr int kExpandMinTokens = 48;

int pick_route(const tbl_latent_mixer& m, int precision, int n_seq, int n_tok) {
    if (precision != TBL_BF16) return kCacheSimt;
    if (n_tok >= kExpandMinTokens && latent_expanded_supported(m)) return kExpanded;
    return latent_tensor_supported(m) ? kCacheTensor : kCacheSimt;
}

int pick_splits(const tbl_latent_mixer& m, int route, int rows, int context) {
    const int tokens = ceil_div(context, 64);                       // a split is worth at least a tile of tokens
    const int units = route == kCacheTensor ? rows * ceil_div(m.heads, latent_tensor_heads(m)) : ceil_div(rows * static_cast<long long>(m.heads), 4);
    int s = units >= kNumSm ? 1 : kNumSm / units;
    if (s > tokens) s = tokens;
    return s < 1 ? 1 : (s > 1024 ? 1024 : s);
}

struct Plan {
    int route, splits;
    size_t cq, q, qa, lat, pm, pl, po, ek, ev, ec, bytes;      // offsets
};

Plan make_plan(const tbl_latent_mixer& m, int precision, int route, int n_seq, int n_tok, int context) {
    Plan w{};
    const size_t rows = static_cast<size_t>(n_seq) * n_tok, e = precision == TBL_BF16 ? 2 : 4;
    w.route = route == kAuto ? pick_route(m, precision, n_seq, n_tok) : route;
    size_t off = 0;
    auto take = [&](size_t bytes) { const size_t at = off; off += round_up(bytes, 256); return at; };
    w.cq = take(e * rows * round_up(m.q_rank, 8));
    w.q = take((w.route == kCacheTensor ? e : sizeof(float)) * rows * m.heads * (m.dim + m.rot_dim));
    w.lat = take(w.route == kCacheTensor ? e * rows * m.heads * m.kv_rank : 0);
    if (w.route == kExpanded) {
        const size_t padded = static_cast<size_t>(n_seq) * latent_expanded_context(context);
        w.ek = take(e * padded * m.heads * m.dim);
        w.ev = take(e * padded * m.heads * m.vdim);
        w.ec = take(e * padded * latent_cache_width(m));
        w.qa = take(e * rows * m.heads * (m.dim + m.rot_dim));
    } else {
        w.splits = pick_splits(m, w.route, static_cast<int>(rows), context);
        w.qa = take(e * rows * m.heads * latent_cache_width(m));
        w.pm = take(sizeof(float) * rows * m.heads * w.splits);
        w.pl = take(sizeof(float) * rows * m.heads * w.splits);
        w.po = take(sizeof(float) * rows * m.heads * w.splits * m.kv_rank);
    }
    w.bytes = off;
    return w;
}

template <typename T>
int run(const tbl_latent_mixer& m, LatentParams p, const Plan& w, int precision, int n_seq, int context, cudaStream_t st) {
    const int rows = n_seq * p.n_tok;
    if (launch_dependent(latent_prep_kernel<T>, dim3(rows), dim3(kPrepThreads), 0, st, p) != cudaSuccess) return TBL_ERR_CUDA;
    DenseCall c{};
    c.x = p.cq; c.w = static_cast<const bf16*>(m.uq.weight); c.bias = m.uq.bias; c.ldx = p.ldq; c.M = rows; c.K = p.q_rank;
    c.N = p.H * (p.d + p.rd); c.ldo = c.N;
    if (w.route == kCacheTensor) c.out_b16 = p.q16; else c.out_f32 = p.q;
    int rc = launch_dense(precision, kDenseAuto, c, st);
    if (rc != TBL_OK) return rc;
    if (w.route == kExpanded) {
        p.context = latent_expanded_context(context);
        return launch_latent_expanded(m, p, n_seq, st);
    }
    if (w.route == kCacheTensor) return launch_latent_tensor(p, rows, st);
    if (launch_dependent(latent_absorb_kernel<T>, dim3(rows, p.H), dim3(128), sizeof(float) * (p.d + p.rd), st, p) != cudaSuccess)
        return TBL_ERR_CUDA;
    rc = launch_simt<T>(p, rows, st);
    if (rc != TBL_OK) return rc;
    return launch_dependent(latent_value_kernel<T>, dim3(rows, p.H), dim3(256), sizeof(float) * (p.R + p.splits), st, p) == cudaSuccess
               ? TBL_OK : TBL_ERR_CUDA;
}

}  // namespace

int check_latent(const tbl_latent_mixer& m, int width) {
    if (m.heads <= 0 || m.heads > 65535 || m.dim <= 0 || m.rot_dim < 2 || m.rot_dim % 2 || m.vdim <= 0 || m.q_rank <= 0 || m.kv_rank <= 0 ||
        m.kv_rank + m.rot_dim > TBL_MAX_LATENT || m.dim + m.rot_dim > 4096 || m.rope_positions <= 0)
        return TBL_ERR_SHAPE;
    if (m.in.inputs != width || m.in.outputs != m.q_rank + m.kv_rank + m.rot_dim + m.heads * m.vdim || m.uq.inputs != m.q_rank ||
        m.uq.outputs != m.heads * (m.dim + m.rot_dim) || m.uk.inputs != m.kv_rank || m.uk.outputs != m.heads * m.dim ||
        m.uv.inputs != m.kv_rank || m.uv.outputs != m.heads * m.vdim || m.out.inputs != m.heads * m.vdim || m.out.outputs != width)
        return TBL_ERR_SHAPE;
    if (!m.in.weight || !m.uq.weight || !m.uk.weight || !m.uv.weight || !m.out.weight || !m.q_norm || !m.kv_norm || !m.rope_cos || !m.rope_sin)
        return TBL_ERR_INVALID_ARG;
    return TBL_OK;
}

int latent_cache_width(const tbl_latent_mixer& m) { return static_cast<int>(round_up(m.kv_rank + m.rot_dim, 8)); }

size_t latent_workspace(const tbl_latent_mixer& m, int precision, int n_seq, int n_tok, int context) {
    return make_plan(m, precision, kAuto, n_seq, n_tok, context).bytes;
}

int launch_latent(const tbl_latent_mixer& m, int precision, int route, float eps, const float* proj, void* cache, int capacity,
                  const int32_t* slots, const int32_t* positions, int n_seq, int n_tok, int context, void* out, void* ws, cudaStream_t st) {
    if (route < kAuto || route > kExpanded) return TBL_ERR_INVALID_ARG;
    if ((route == kCacheTensor && (precision != TBL_BF16 || !latent_tensor_supported(m))) ||
        (route == kExpanded && (precision != TBL_BF16 || !latent_expanded_supported(m))))
        return TBL_ERR_SHAPE;
    const Plan w = make_plan(m, precision, route, n_seq, n_tok, context);
    uint8_t* base = static_cast<uint8_t*>(ws);
    LatentParams p{};
    p.proj = proj; p.q_norm = m.q_norm; p.kv_norm = m.kv_norm; p.rope_cos = m.rope_cos; p.rope_sin = m.rope_sin;
    p.uk = static_cast<const bf16*>(m.uk.weight); p.uk_t = static_cast<const bf16*>(m.uk_t); p.uv = static_cast<const bf16*>(m.uv.weight);
    p.cache = cache; p.slots = slots; p.positions = positions; p.out = out; p.status = device_status_ptr();
    if (!p.status) return TBL_ERR_CUDA;
    p.cq = base + w.cq; p.q = reinterpret_cast<float*>(base + w.q); p.q16 = reinterpret_cast<bf16*>(base + w.q); p.lat = reinterpret_cast<bf16*>(base + w.lat); p.qa = base + w.qa;
    p.part_m = reinterpret_cast<float*>(base + w.pm); p.part_l = reinterpret_cast<float*>(base + w.pl);
    p.part_o = reinterpret_cast<float*>(base + w.po);
    p.keys = reinterpret_cast<bf16*>(base + w.ek); p.values = reinterpret_cast<bf16*>(base + w.ev);
    p.gathered = reinterpret_cast<bf16*>(base + w.ec);
    p.ld = m.in.outputs; p.ldq = static_cast<int>(round_up(m.q_rank, 8)); p.cw = latent_cache_width(m);
    p.H = m.heads; p.d = m.dim; p.rd = m.rot_dim; p.vd = m.vdim; p.R = m.kv_rank; p.q_rank = m.q_rank;
    p.capacity = capacity; p.rope_positions = m.rope_positions; p.n_tok = n_tok; p.splits = w.splits; p.context = context;
    p.scale = m.scale; p.eps = eps;
    return precision == TBL_BF16 ? run<bf16>(m, p, w, precision, n_seq, context, st) : run<float>(m, p, w, precision, n_seq, context, st);
}

}  // namespace stack
}  // namespace tbl

using namespace tbl;
using namespace tbl::stack;

extern "C" {

size_t tbl_latent_workspace_bytes(const tbl_latent_mixer* mixer, int precision, int n_seq, int n_tok, int context) {
    if (!mixer || n_seq <= 0 || n_tok <= 0 || context <= 0 || check_latent(*mixer, mixer->in.inputs) != TBL_OK) return 0;
    size_t most = 0;
    for (int route = kAuto; route <= kExpanded; ++route) {
        const size_t b = make_plan(*mixer, precision, route, n_seq, n_tok, context).bytes;
        most = b > most ? b : most;
    }
    return most;
}

int tbl_latent_forward(const tbl_latent_mixer* mixer, int precision, int route, float eps, const float* proj_dev, void* cache_dev,
                       int capacity, const int32_t* slots_dev, const int32_t* positions_dev, int n_seq, int n_tok, int context,
                       void* out_dev, void* workspace_dev, size_t workspace_bytes, void* stream) {
    if (!mixer || !proj_dev || !cache_dev || !slots_dev || !positions_dev || !out_dev || n_seq <= 0 || n_tok <= 0 || capacity <= 0 ||
        context < n_tok || context > capacity || (precision != TBL_F32 && precision != TBL_BF16))
        return TBL_ERR_INVALID_ARG;
    const int rc = check_latent(*mixer, mixer->in.inputs);
    if (rc != TBL_OK) return rc;
    if (!workspace_dev || workspace_bytes < tbl_latent_workspace_bytes(mixer, precision, n_seq, n_tok, context)) return TBL_ERR_WORKSPACE;
    if ((reinterpret_cast<uintptr_t>(workspace_dev) & 255) || (reinterpret_cast<uintptr_t>(cache_dev) & 15)) return TBL_ERR_ALIGNMENT;
    return launch_latent(*mixer, precision, route, eps, proj_dev, cache_dev, capacity, slots_dev, positions_dev, n_seq, n_tok, context,
                         out_dev, workspace_dev, static_cast<cudaStream_t>(stream));
}

}  // extern "C"
