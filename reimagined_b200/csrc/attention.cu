// Softmax attention with grouped key/value heads and, optionally, two maps per head (differential attention).
//
//   attention_prep_kernel    appends a portion's keys and values to the cache; queries in bf16 for the flash kernel
//   attention_simt_kernel    any sizes, fp32 arithmetic; split over the context
//   attention_merge_kernel   brings the splits together, combines the maps, head norm, output gate
// The kernels that stream the cache for a few query rows and the flash kernel for prompts are in attention_decode.cu and
// attention_prefill.cu.  Scores, softmax weights and their sums are fp32 throughout.
#include "attention.cuh"

namespace tbl {
namespace stack {
namespace {

constexpr int kPrepThreads = 256;

// eight neighbouring numbers of a row of fp32 projections
__device__ __forceinline__ void load8(const float* src, int n, bool vec, float (&v)[8]) {
    if (vec && n >= 8) {
        const float4 a = *reinterpret_cast<const float4*>(src), b = *reinterpret_cast<const float4*>(src + 4);
        v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
    } else {
#pragma unroll
        for (int i = 0; i < 8; ++i) v[i] = i < n ? src[i] : 0.0f;
    }
}
__device__ __forceinline__ void store8(bf16* dst, const float (&v)[8]) {
    *reinterpret_cast<uint4*>(dst) = make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
}
__device__ __forceinline__ void store8(float* dst, const float (&v)[8]) {
    *reinterpret_cast<float4*>(dst) = make_float4(v[0], v[1], v[2], v[3]);
    *reinterpret_cast<float4*>(dst + 4) = make_float4(v[4], v[5], v[6], v[7]);
}

// One CTA per row of the step; a thread takes eight neighbouring numbers at a time (the padded parts are multiples of 16).
template <typename T>
__global__ void __launch_bounds__(kPrepThreads) attention_prep_kernel(const AttnParams p) {
    pdl_launch_dependents();
    pdl_wait();
    const int row = blockIdx.x, tid = threadIdx.x;
    const int slot = p.slots[row / p.n_tok], pos = p.positions[slot] + row % p.n_tok;
    const float* pr = p.proj + static_cast<size_t>(row) * p.ld;
    float v[8];
    if (p.q16) {
        const float t = temperature_of(p, pos);
        const int per = p.dp / 8, n = p.H * p.maps * per;
        bf16* out = p.q16 + static_cast<size_t>(row) * p.H * p.maps * p.dp;
        for (int i = tid; i < n; i += kPrepThreads) {
            const int head = i / per, c = (i - head * per) * 8;
            load8(pr + head * p.d + c, p.d - c, p.vec, v);
#pragma unroll
            for (int e = 0; e < 8; ++e) v[e] *= t;
            store8(out + i * 8, v);
        }
    }
    if (!p.append) return;
    if (pos < 0 || pos >= p.capacity || (p.temperature && pos >= p.temperature_positions)) {
        if (tid == 0) atomicOr(p.status, TBL_DEV_CACHE_FULL);
        return;
    }
    const int per = p.cw / 8, kper = p.dp / 8, keys = p.maps * kper;
    for (int i = tid; i < p.G * per; i += kPrepThreads) {
        const int g = i / per, c = i - g * per;
        if (c < keys) {
            const int map = c / kper, e = (c - map * kper) * 8;
            load8(pr + p.k_off + (g * p.maps + map) * p.d + e, p.d - e, p.vec, v);
        } else {
            const int e = (c - keys) * 8;
            load8(pr + p.v_off + g * p.vd + e, p.vd - e, p.vec, v);
        }
        store8(static_cast<T*>(p.cache) + cache_row(p, slot, g, pos) + c * 8, v);
    }
}

// ---- SIMT ---------------------------------------------------------------------------------------------------------------
// A CTA: 16 query rows of a (sequence, kv head, map), one split of the context, 32 tokens at a time.  NV: value columns per
// thread (16 threads share a row).
constexpr int kSimtRows = 16, kSimtTokens = 32, kSimtThreads = 256;

size_t simt_smem(int d, int vd) {
    return sizeof(float) * (static_cast<size_t>(kSimtRows + kSimtTokens) * (d + 1) + static_cast<size_t>(kSimtTokens) * vd);
}

template <typename T, int NV>
__global__ void __launch_bounds__(kSimtThreads) attention_simt_kernel(const AttnParams p) {
    extern __shared__ float sm[];
    __shared__ float s_s[kSimtRows][kSimtTokens + 1], m_s[kSimtRows], l_s[kSimtRows], f_s[kSimtRows];
    const int ld = p.d + 1;
    float* q_s = sm;                             // [16][ld]
    float* k_s = q_s + kSimtRows * ld;           // [32][ld]
    float* v_s = k_s + kSimtTokens * ld;         // [32][vd]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int unit = blockIdx.y, map = unit % p.maps, g = unit / p.maps % p.G, seq = unit / (p.maps * p.G), split = blockIdx.z;
    pdl_launch_dependents();
    pdl_wait();
    const int first = blockIdx.x * kSimtRows, total = p.n_tok * p.group;
    const int slot = p.slots[seq], pos0 = p.positions[slot];
    const int n = min(pos0 + min(total - 1, first + kSimtRows - 1) / p.group + 1, p.capacity);     // tokens the last row sees
    const int per = (n + p.splits - 1) / p.splits;
    const int t0 = min(split * per, n), t1 = min(n, t0 + per);
    for (int i = tid; i < kSimtRows * p.d; i += kSimtThreads) {
        const int r = i / p.d, c = i - r * p.d, at = first + r;
        float q = 0.0f;
        if (at < total) {
            const int t = at / p.group, head = g * p.group + at % p.group;
            q = p.proj[(static_cast<size_t>(seq) * p.n_tok + t) * p.ld + (head * p.maps + map) * p.d + c] * temperature_of(p, pos0 + t);
        }
        q_s[r * ld + c] = q;
    }
    if (tid < kSimtRows) { m_s[tid] = -INFINITY; l_s[tid] = 0.0f; }
    float acc[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) acc[i] = 0.0f;
    const int row = tid >> 4, col = tid & 15;
    const int last = pos0 + min(first + row, total - 1) / p.group;           // last visible token of this thread's row
    const T* cache = static_cast<const T*>(p.cache) + cache_row(p, slot, g, 0);
    for (int t = t0; t < t1; t += kSimtTokens) {
        __syncthreads();
        for (int i = tid; i < kSimtTokens * p.d; i += kSimtThreads) {
            const int r = i / p.d, c = i - r * p.d;
            k_s[r * ld + c] = t + r < t1 ? to_f(cache[static_cast<size_t>(t + r) * p.cw + map * p.dp + c]) : 0.0f;
        }
        for (int i = tid; i < kSimtTokens * p.vd; i += kSimtThreads) {
            const int r = i / p.vd, c = i - r * p.vd;
            v_s[i] = t + r < t1 ? to_f(cache[static_cast<size_t>(t + r) * p.cw + p.maps * p.dp + c]) : 0.0f;
        }
        __syncthreads();
        float a = 0.0f, b = 0.0f;
        const float *qr = q_s + row * ld, *ka = k_s + col * ld, *kb = ka + 16 * ld;
#pragma unroll 4
        for (int c = 0; c < p.d; ++c) { a = fmaf(qr[c], ka[c], a); b = fmaf(qr[c], kb[c], b); }
        s_s[row][col] = t + col <= min(last, t1 - 1) ? a * p.scale_log2 : -INFINITY;
        s_s[row][col + 16] = t + col + 16 <= min(last, t1 - 1) ? b * p.scale_log2 : -INFINITY;
        __syncthreads();
#pragma unroll
        for (int i = 0; i < kSimtRows / 8; ++i) {
            const int r = warp * (kSimtRows / 8) + i;
            const float x = s_s[r][lane], mo = m_s[r], mn = fmaxf(mo, warp_max(x));
            // a row that has seen nothing yet keeps its maximum at -infinity and its weights at zero
            const float w = mn == -INFINITY ? 0.0f : exp2f(x - mn), sum = warp_sum(w);
            s_s[r][lane] = w;
            __syncwarp();
            if (lane == 0) {
                const float f = mo == -INFINITY ? 0.0f : exp2f(mo - mn);
                f_s[r] = f;
                m_s[r] = mn;
                l_s[r] = fmaf(l_s[r], f, sum);
            }
        }
        __syncthreads();
        const float f = f_s[row];
#pragma unroll
        for (int i = 0; i < NV; ++i) acc[i] *= f;
        for (int k = 0; k < kSimtTokens; ++k) {
            const float w = s_s[row][k];
#pragma unroll
            for (int i = 0; i < NV; ++i)
                if (col + 16 * i < p.vd) acc[i] = fmaf(w, v_s[k * p.vd + col + 16 * i], acc[i]);
        }
    }
    __syncthreads();
    if (first + row >= total) return;
    const int t = (first + row) / p.group, head = g * p.group + (first + row) % p.group;
    const size_t u = (((static_cast<size_t>(seq) * p.n_tok + t) * p.H + head) * p.maps + map) * p.splits + split;
#pragma unroll
    for (int i = 0; i < NV; ++i)
        if (col + 16 * i < p.vd) p.part_o[u * p.vp + col + 16 * i] = acc[i];
    if (col == 0) { p.part_m[u] = m_s[row]; p.part_l[u] = l_s[row]; }
}

// ---- merge ----------------------------------------------------------------------------------------------------------------
// One CTA per (row, head).  128 threads share a map's value columns; of a layer with one map the second half of the CTA
// takes every other split.
constexpr int kMergeThreads = 256, kMergeMaxSplits = 1024;

template <typename T>
__global__ void __launch_bounds__(kMergeThreads) attention_merge_kernel(const AttnParams p) {
    __shared__ float fac[2][kMergeMaxSplits], inv_s[2], red[kMergeThreads / 32], part[2][TBL_MAX_ATTENTION_DIM];
    pdl_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int row = blockIdx.x, head = blockIdx.y;
    pdl_wait();
    const size_t unit = (static_cast<size_t>(row) * p.H + head) * p.maps * p.splits;
    if (warp < p.maps) {
        const float *pm = p.part_m + unit + warp * p.splits, *pl = p.part_l + unit + warp * p.splits;
        float m = -INFINITY, l = 0.0f;
        for (int s = lane; s < p.splits; s += 32) m = fmaxf(m, pm[s]);
        m = warp_max(m);
        for (int s = lane; s < p.splits; s += 32) {
            const float ms = pm[s], f = ms == -INFINITY ? 0.0f : exp2f(ms - m);
            fac[warp][s] = f;
            l = fmaf(pl[s], f, l);
        }
        l = warp_sum(l);
        if (lane == 0) inv_s[warp] = (warp == 0 ? 1.0f : -p.lambda) / l;
    }
    __syncthreads();
    const int half = tid >> 7, map = p.maps == 2 ? half : 0, s0 = p.maps == 2 ? 0 : half, step = p.maps == 2 ? 1 : 2;
    for (int c = tid & 127; c < p.vd; c += 128) {
        const float* o = p.part_o + (unit + map * p.splits) * p.vp + c;
        float v = 0.0f;
#pragma unroll 8
        for (int s = s0; s < p.splits; s += step) v = fmaf(o[static_cast<size_t>(s) * p.vp], fac[map][s], v);
        part[half][c] = v * inv_s[map];
    }
    __syncthreads();
    float ss = 0.0f;
    for (int c = tid; c < p.vd; c += kMergeThreads) {
        const float v = part[0][c] + part[1][c];
        part[0][c] = v;                          // its only reader and writer from here on
        ss = fmaf(v, v, ss);
    }
    float f = 1.0f;
    if (p.maps == 2) {
        ss = warp_sum(ss);
        if (lane == 0) red[warp] = ss;
        __syncthreads();
        float total = 0.0f;
#pragma unroll
        for (int w = 0; w < kMergeThreads / 32; ++w) total += red[w];
        f = p.out_scale / sqrtf(total / static_cast<float>(p.vd) + p.eps);
    }
    const float* gate = p.g_off < 0 ? nullptr : p.proj + static_cast<size_t>(row) * p.ld + p.g_off + head * p.vd;
    T* out = static_cast<T*>(p.out) + (static_cast<size_t>(row) * p.H + head) * p.vd;
    for (int c = tid; c < p.vd; c += kMergeThreads) out[c] = from_f<T>(part[0][c] * f * (gate ? sigmoid_f(gate[c]) : 1.0f));
}

template <typename T, int NV>
int launch_simt_nv(const AttnParams& p, int n_seq, cudaStream_t st) {
    static bool done[64] = {};
    const size_t smem = simt_smem(p.d, p.vd);
    if (smem > 200 * 1024) return TBL_ERR_SHAPE;
    if (allow_smem(attention_simt_kernel<T, NV>, smem, done) != cudaSuccess) return TBL_ERR_CUDA;
    const dim3 grid(ceil_div(static_cast<long long>(p.n_tok) * p.group, kSimtRows), n_seq * p.G * p.maps, p.splits);
    if (grid.y > 65535) return TBL_ERR_SHAPE;
    return launch_dependent(attention_simt_kernel<T, NV>, grid, dim3(kSimtThreads), smem, st, p) == cudaSuccess ? TBL_OK : TBL_ERR_CUDA;
}

template <typename T>
int launch_simt(const AttnParams& p, int n_seq, cudaStream_t st) {
    if (p.vd <= 64) return launch_simt_nv<T, 4>(p, n_seq, st);
    if (p.vd <= 128) return launch_simt_nv<T, 8>(p, n_seq, st);
    if (p.vd <= 256) return launch_simt_nv<T, 16>(p, n_seq, st);
    return launch_simt_nv<T, 32>(p, n_seq, st);
}

enum Route { kAuto = 0, kSimt = 1, kStream = 2, kFlash = 3 };
constexpr int kFlashMinTokens = 48;

int pick_route(const tbl_attention_mixer& m, int precision, int n_tok) {
    if (precision != TBL_BF16) return kSimt;
    if (n_tok >= kFlashMinTokens && attention_flash_supported(m)) return kFlash;
    return attention_stream_supported(m) ? kStream : kSimt;
}

int pick_splits(const tbl_attention_mixer& m, int route, int n_seq, int n_tok, int context) {
    if (route == kFlash) return 1;
    const long long blocks = ceil_div(static_cast<long long>(n_tok) * (m.heads / m.kv_heads), 16);
    const long long units = blocks * n_seq * m.kv_heads * (route == kSimt ? m.maps : 1);
    const int tokens = ceil_div(context, 64);                       // a split is worth at least a tile of tokens
    long long s = 2LL * kNumSm / units;
    if (s > tokens) s = tokens;
    // a cluster's worth is enough when that keeps most of the SMs busy, or leaves a CTA little to read
    if (route == kStream && s > kClusterSplits && (units * kClusterSplits >= kNumSm / 2 || tokens <= 8 * kClusterSplits)) s = kClusterSplits;
    return s < 1 ? 1 : (s > kMergeMaxSplits ? kMergeMaxSplits : static_cast<int>(s));
}

struct Plan {
    int route, splits, fused_append;
    size_t q16, pm, pl, po, bytes;             // offsets
};

int padded(int n) { return static_cast<int>(round_up(n, 16)); }

Plan make_plan(const tbl_attention_mixer& m, int precision, int route, int n_seq, int n_tok, int context) {
    Plan w{};
    const size_t rows = static_cast<size_t>(n_seq) * n_tok;
    w.route = route == kAuto ? pick_route(m, precision, n_tok) : route;
    w.splits = pick_splits(m, w.route, n_seq, n_tok, context);
    // one token per sequence and one block of query rows: the CTA whose split holds the token appends it
    w.fused_append = w.route == kStream && n_tok == 1 && m.heads / m.kv_heads <= 16;
    size_t off = 0;
    auto take = [&](size_t bytes) { const size_t at = off; off += round_up(bytes, 256); return at; };
    const size_t units = rows * m.heads * m.maps * w.splits;
    w.q16 = take(w.route == kFlash ? 2 * rows * m.heads * m.maps * padded(m.dim) : 0);
    const bool parts = w.route == kSimt || (w.route == kStream && w.splits > kClusterSplits) || (w.route == kFlash && !attention_flash_whole(m));
    w.pm = take(parts ? sizeof(float) * units : 0);
    w.pl = take(parts ? sizeof(float) * units : 0);
    w.po = take(parts ? sizeof(float) * units * padded(m.vdim) : 0);
    w.bytes = off;
    return w;
}

template <typename T>
int run(const tbl_attention_mixer& m, AttnParams p, const Plan& w, int n_seq, cudaStream_t st) {
    const int rows = n_seq * p.n_tok;
    const bool append = m.kv_from < 0;
    bf16* q16 = p.q16;
    p.q16 = w.route == kFlash ? q16 : nullptr;
    p.append = append && !w.fused_append;
    if (p.append || p.q16) {
        if (launch_dependent(attention_prep_kernel<T>, dim3(rows), dim3(kPrepThreads), 0, st, p) != cudaSuccess) return TBL_ERR_CUDA;
    }
    p.append = append && w.fused_append;
    int rc;
    bool merge = w.route == kSimt || w.splits > kClusterSplits;
    if (w.route == kFlash) {
        rc = launch_attention_flash(p, n_seq, st);
        merge = !attention_flash_whole(m);
    } else if (w.route == kStream) {
        rc = launch_attention_stream(p, n_seq, st);
    } else {
        rc = launch_simt<T>(p, n_seq, st);
    }
    if (rc != TBL_OK || !merge) return rc;
    return launch_dependent(attention_merge_kernel<T>, dim3(rows, p.H), dim3(kMergeThreads), 0, st, p) == cudaSuccess ? TBL_OK : TBL_ERR_CUDA;
}

}  // namespace

int check_attention(const tbl_attention_mixer& m, int width) {
    if (m.heads <= 0 || m.kv_heads <= 0 || m.heads > 65535 || m.heads % m.kv_heads || m.dim <= 0 || m.vdim <= 0 ||
        m.dim > TBL_MAX_ATTENTION_DIM || m.vdim > TBL_MAX_ATTENTION_DIM || (m.maps != 1 && m.maps != 2) ||
        (m.temperature && m.temperature_positions <= 0))
        return TBL_ERR_SHAPE;
    const int kv = m.kv_from < 0 ? m.kv_heads * (m.maps * m.dim + m.vdim) : 0;
    if (m.in.inputs != width || m.in.outputs != m.heads * m.maps * m.dim + kv + (m.gated ? m.heads * m.vdim : 0) ||
        m.out.inputs != m.heads * m.vdim || m.out.outputs != width)
        return TBL_ERR_SHAPE;
    return m.in.weight && m.out.weight ? TBL_OK : TBL_ERR_INVALID_ARG;
}

int attention_cache_width(const tbl_attention_mixer& m) { return m.maps * padded(m.dim) + padded(m.vdim); }

size_t attention_workspace(const tbl_attention_mixer& m, int precision, int n_seq, int n_tok, int context) {
    return make_plan(m, precision, kAuto, n_seq, n_tok, context).bytes;
}

int launch_attention(const tbl_attention_mixer& m, int precision, int route, float eps, const float* proj, void* cache, int n_slots,
                     int capacity, const int32_t* slots, const int32_t* positions, int n_seq, int n_tok, int context, void* out,
                     void* ws, cudaStream_t st) {
    if (route < kAuto || route > kFlash) return TBL_ERR_INVALID_ARG;
    if ((route == kStream && (precision != TBL_BF16 || !attention_stream_supported(m))) ||
        (route == kFlash && (precision != TBL_BF16 || !attention_flash_supported(m))))
        return TBL_ERR_SHAPE;
    const Plan w = make_plan(m, precision, route, n_seq, n_tok, context);
    uint8_t* base = static_cast<uint8_t*>(ws);
    AttnParams p{};
    p.status = device_status_ptr();
    if (!p.status) return TBL_ERR_CUDA;
    p.proj = proj; p.temperature = m.temperature; p.temperature_positions = m.temperature_positions; p.cache = cache;
    p.slots = slots; p.positions = positions; p.out = out;
    p.q16 = reinterpret_cast<bf16*>(base + w.q16); p.part_m = reinterpret_cast<float*>(base + w.pm);
    p.part_l = reinterpret_cast<float*>(base + w.pl); p.part_o = reinterpret_cast<float*>(base + w.po);
    p.ld = m.in.outputs; p.k_off = m.heads * m.maps * m.dim;
    p.v_off = p.k_off + (m.kv_from < 0 ? m.kv_heads * m.maps * m.dim : 0);
    p.g_off = m.gated ? p.v_off + (m.kv_from < 0 ? m.kv_heads * m.vdim : 0) : -1;
    p.H = m.heads; p.G = m.kv_heads; p.group = m.heads / m.kv_heads; p.maps = m.maps; p.d = m.dim; p.vd = m.vdim;
    p.dp = padded(m.dim); p.vp = padded(m.vdim); p.cw = attention_cache_width(m);
    p.n_slots = n_slots; p.capacity = capacity; p.n_tok = n_tok; p.splits = w.splits;
    p.vec = (p.ld | m.dim | m.vdim) % 4 == 0 && (reinterpret_cast<uintptr_t>(proj) & 15) == 0;
    p.scale_log2 = static_cast<float>(static_cast<double>(m.scale) * 1.4426950408889634); p.lambda = m.lambda; p.out_scale = m.out_scale; p.eps = eps;
    return precision == TBL_BF16 ? run<bf16>(m, p, w, n_seq, st) : run<float>(m, p, w, n_seq, st);
}

}  // namespace stack
}  // namespace tbl

using namespace tbl;
using namespace tbl::stack;

extern "C" {

int tbl_attention_cache_width(const tbl_attention_mixer* mixer) {
    return mixer && check_attention(*mixer, mixer->in.inputs) == TBL_OK ? attention_cache_width(*mixer) : 0;
}

size_t tbl_attention_workspace_bytes(const tbl_attention_mixer* mixer, int precision, int n_seq, int n_tok, int context) {
    if (!mixer || n_seq <= 0 || n_tok <= 0 || context <= 0 || check_attention(*mixer, mixer->in.inputs) != TBL_OK) return 0;
    size_t most = 0;
    for (int route = kAuto; route <= kFlash; ++route) {
        const size_t b = make_plan(*mixer, precision, route, n_seq, n_tok, context).bytes;
        most = b > most ? b : most;
    }
    return most > 0 ? most : 256;
}

int tbl_attention_forward(const tbl_attention_mixer* mixer, int precision, int route, float eps, const float* proj_dev, void* cache_dev,
                          int slots, int capacity, const int32_t* slots_dev, const int32_t* positions_dev, int n_seq, int n_tok,
                          int context, void* out_dev, void* workspace_dev, size_t workspace_bytes, void* stream) {
    if (!mixer || !proj_dev || !cache_dev || !slots_dev || !positions_dev || !out_dev || n_seq <= 0 || n_tok <= 0 || slots < n_seq ||
        capacity <= 0 || context < n_tok || context > capacity || (precision != TBL_F32 && precision != TBL_BF16))
        return TBL_ERR_INVALID_ARG;
    const int rc = check_attention(*mixer, mixer->in.inputs);
    if (rc != TBL_OK) return rc;
    if (!workspace_dev || workspace_bytes < tbl_attention_workspace_bytes(mixer, precision, n_seq, n_tok, context)) return TBL_ERR_WORKSPACE;
    if ((reinterpret_cast<uintptr_t>(workspace_dev) & 255) || (reinterpret_cast<uintptr_t>(cache_dev) & 15)) return TBL_ERR_ALIGNMENT;
    return launch_attention(*mixer, precision, route, eps, proj_dev, cache_dev, slots, capacity, slots_dev, positions_dev, n_seq, n_tok,
                            context, out_dev, workspace_dev, static_cast<cudaStream_t>(stream));
}

}  // extern "C"
