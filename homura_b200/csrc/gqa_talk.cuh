// Attention whose heads mix their scores (GqaAttnArgs::talk): part of gqa_attn.cu.
//
// A CTA takes all heads of a tile of rows (rows of a run that follow one another; a decoded token is a tile of one) and a share of
// their pages.  A page comes block by block through a ring of bulk copies: the keys of every key head, then the values of every one.
//   scores^T [16 tokens x pairs] = K [16 x dim] . Q^T     per key head, into shared memory
//   mix, mask, softmax                                    per (row, head): lanes along the tokens, f32
//   out^T    [16 values x pairs] += V^T [16 x 64] . P^T   per key head, accumulators in shared memory
// A pair is a (row, head); those of a key head are the MMAs' columns, eight at a time.  Queries and weights are three bf16 terms each.

constexpr int TALK_MAX_STAGES = 16;
constexpr int TALK_RAW_LD = GQA_PAGE + 4, TALK_P_LD = GQA_PAGE + 8;  // row strides of scores (floats) and weights (bf16): no bank conflicts

struct TalkGeom {
    int rows;       // of a tile
    int per;        // pairs of a key head: rows * heads per key head
    int ntile;      // tiles of eight of them
    int cols2;      // pairs of columns that a tile uses (accumulators of the others are not kept)
    int stages;
    uint32_t block; // bytes of a ring stage
    size_t front;   // bytes of the ring, which takes the results afterwards
    size_t q, raw, p, corr, o, ml, talk, recv, pages, qi, pair, smem;  // offsets from the front's end, total
};

inline bool talk_geom(const GqaAttnArgs& a, int rows, int nsplit, int pages_per_cta, size_t most, TalkGeom* g) {
    const int H = a.heads, G = a.pool.kv_heads, gq = H / G, dp = gqa_pad(a.pool.dim), vp = gqa_pad(a.pool.vdim);
    const size_t pairs = (size_t)rows * H, padded = pairs + 8;
    g->rows = rows;
    g->per = rows * gq;
    g->ntile = (g->per + 7) / 8;
    g->cols2 = g->per >= 8 ? 4 : (g->per + 1) / 2;
    g->block = (uint32_t)(GQA_PAGE * std::max(dp, vp) * 2);
    size_t at = 0;
    auto take = [&](size_t bytes) {
        const size_t first = at;
        at += (bytes + 15) / 16 * 16;
        return first;
    };
    g->q = take(3 * padded * (dp + 8) * 2);
    g->raw = take(pairs * TALK_RAW_LD * 4);
    g->p = take(3 * padded * TALK_P_LD * 2);
    g->corr = take(padded * 4);
    g->o = take((size_t)G * (vp / 16) * g->ntile * g->cols2 * 8 * 16);
    g->ml = take(pairs * 8);
    g->talk = take((size_t)H * ((H + 3) / 4 * 4) * 4);
    // what a CTA receives: from every split, its share of the pairs (values, maximum, sum)
    g->recv = take(nsplit > 1 ? nsplit * ((pairs + nsplit - 1) / nsplit) * (vp + 4) * 4 : 0);
    g->pages = take((size_t)pages_per_cta * 4);
    g->qi = take(pairs * 2);
    g->pair = take((size_t)g->per * 2);
    const size_t result = pairs * (vp + 4) * 4;
    if (at + std::max(result, 2 * (size_t)g->block) + 128 > most) return false;
    g->stages = (int)std::min<size_t>({(most - at - 128) / g->block, (size_t)TALK_MAX_STAGES, (size_t)2 * G * std::max(1, pages_per_cta)});
    g->front = (std::max(result, (size_t)g->stages * g->block) + 127) / 128 * 128;
    g->smem = g->front + at;
    return g->smem <= most;
}

// Scores of KH heads of a row out of all heads' (x: this lane's two tokens of the row's first head), mask, running softmax, weights.
template <int KH>
__device__ __forceinline__ void talk_mix(const GqaAttnArgs& a, int r, int h0, int pos, int from, int ta, const float* x, const float* tk, int HP, const uint16_t* qi, uint16_t* ps, int padded, float* ml, float* corr) {
    const int H = a.heads, lane = threadIdx.x & 31;
    float2 s[KH];
    float old[KH];
#pragma unroll
    for (int k = 0; k < KH; ++k) {
        s[k] = make_float2(0.f, 0.f);
        old[k] = h0 + k < H ? ml[2 * (r * H + h0 + k)] : 0.f;
    }
#pragma unroll 4
    for (int e = 0; e < H; ++e) {
        const float2 v = *reinterpret_cast<const float2*>(x + e * TALK_RAW_LD);
        float t[KH];
        if constexpr (KH == 4) {
            const float4 w = *reinterpret_cast<const float4*>(tk + e * HP + h0);
            t[0] = w.x; t[1] = w.y; t[2] = w.z; t[3] = w.w;
        } else if constexpr (KH == 2) {
            const float2 w = *reinterpret_cast<const float2*>(tk + e * HP + h0);
            t[0] = w.x; t[1] = w.y;
        } else {
            t[0] = tk[e * HP + h0];
        }
#pragma unroll
        for (int k = 0; k < KH; ++k) {
            s[k].x = fmaf(t[k], v.x, s[k].x);
            s[k].y = fmaf(t[k], v.y, s[k].y);
        }
    }
    const bool va = ta <= pos && (ta >= from || ta < a.keep_first), vb = ta + 1 <= pos && (ta + 1 >= from || ta + 1 < a.keep_first);
    float mx[KH], sum[KH], f[KH];
#pragma unroll
    for (int k = 0; k < KH; ++k) {
        s[k].x = va ? s[k].x : -INFINITY;
        s[k].y = vb ? s[k].y : -INFINITY;
        mx[k] = fmaxf(s[k].x, s[k].y);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1)
#pragma unroll
        for (int k = 0; k < KH; ++k) mx[k] = fmaxf(mx[k], __shfl_xor_sync(0xffffffffu, mx[k], o));
#pragma unroll
    for (int k = 0; k < KH; ++k) {
        mx[k] = fmaxf(old[k], mx[k]);
        const float ref = mx[k] == -INFINITY ? 0.f : mx[k];  // no token of this pair yet
        f[k] = exp2f(old[k] - ref);
        s[k].x = exp2f(s[k].x - ref);
        s[k].y = exp2f(s[k].y - ref);
        sum[k] = s[k].x + s[k].y;
        if (h0 + k < H) {
            uint32_t t[3];
            bf16x2_split3(s[k].x, s[k].y, t[0], t[1], t[2]);
            uint16_t* dst = ps + (size_t)qi[r * H + h0 + k] * TALK_P_LD + 2 * lane;
#pragma unroll
            for (int e = 0; e < 3; ++e) *reinterpret_cast<uint32_t*>(dst + (size_t)e * padded * TALK_P_LD) = t[e];
        }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1)
#pragma unroll
        for (int k = 0; k < KH; ++k) sum[k] += __shfl_xor_sync(0xffffffffu, sum[k], o);
    if (lane < KH && h0 + lane < H) {
        float m = mx[0], c = f[0], l = sum[0];
#pragma unroll
        for (int k = 1; k < KH; ++k)
            if (lane == k) {
                m = mx[k];
                c = f[k];
                l = sum[k];
            }
        float* d = ml + 2 * (r * H + h0 + lane);
        d[0] = m;
        d[1] = fmaf(d[1], c, l);
        corr[qi[r * H + h0 + lane]] = c;
    }
    __syncwarp();
}

__global__ void __launch_bounds__(B_THREADS, 2) talk_attn_mma_kernel(const __grid_constant__ GqaAttnArgs a, const __grid_constant__ TalkGeom geo) {
    extern __shared__ __align__(128) unsigned char dyn[];
    const int H = a.heads, G = a.pool.kv_heads, gq = H / G, dim = a.pool.dim, vdim = a.pool.vdim, dp = gqa_pad(dim), vp = gqa_pad(vdim), kt_n = dp / 16, vt_n = vp / 16, ldo = vp + 4;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, split = blockIdx.x, NST = geo.stages, HP = (H + 3) & ~3;
    unsigned char *ring = dyn, *back = dyn + geo.front;
    const int padded = geo.rows * H + 8, ldq = dp + 8;
    uint16_t* qs = reinterpret_cast<uint16_t*>(back + geo.q);        // [3][padded][ldq], pairs by key head
    float* raw = reinterpret_cast<float*>(back + geo.raw);           // [row][head][TALK_RAW_LD]
    uint16_t* ps = reinterpret_cast<uint16_t*>(back + geo.p);        // [3][padded][TALK_P_LD], pairs by key head
    float* corr = reinterpret_cast<float*>(back + geo.corr);         // [padded]
    float4* os = reinterpret_cast<float4*>(back + geo.o);            // [key head][16 values][tile of pairs][two columns][8 lanes]
    float* ml = reinterpret_cast<float*>(back + geo.ml);             // [row][head][2]
    float* tk = reinterpret_cast<float*>(back + geo.talk);           // [head that is read][head, padded]
    float* recv = reinterpret_cast<float*>(back + geo.recv);         // [split][pairs of this CTA][vp + 4]
    int32_t* pt_s = reinterpret_cast<int32_t*>(back + geo.pages);
    uint16_t* qi = reinterpret_cast<uint16_t*>(back + geo.qi);       // [row][head] -> pair by key head
    uint16_t* pair = reinterpret_cast<uint16_t*>(back + geo.pair);   // pair of the first key head -> [row][head]
    __shared__ uint64_t full[TALK_MAX_STAGES], empty[TALK_MAX_STAGES], s_rbar;
    __shared__ volatile int s_abort;

    int row0 = blockIdx.z, rows = 1;
    if (a.runs.n > 0) {
        int r = 0;
        while (r + 1 < a.runs.n && a.runs.tile[r + 1] <= blockIdx.z) ++r;
        row0 = a.runs.row[r] + (blockIdx.z - a.runs.tile[r]) * geo.rows;
        rows = min(geo.rows, a.runs.row[r + 1] - row0);
    }
    const int pairs = rows * H;
    // the splits of a tile share its pairs: pair p is combined and stored by split p % ns
    const int ns = a.nsplit, rank = ns > 1 ? (int)cluster_ctarank() : 0, own = pairs > rank ? (pairs - rank + ns - 1) / ns : 0, own_most = (geo.rows * H + ns - 1) / ns;
    if (tid < NST) {
        mb_init(&full[tid], 1);
        mb_init(&empty[tid], ATT_WARPS);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (tid == 0) {
        s_abort = 0;
        mb_init(&s_rbar, 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        if (ns > 1 && own > 0) mb_expect_tx(&s_rbar, (uint32_t)((ns - 1) * own * (vp + 2) * 4));
    }
    pdl_launch_dependents();
    if (ns > 1) {
        cluster_arrive_release();
        cluster_wait_acquire();
    }
    // positions, pages and the mixing matrix do not depend on the launch in front
    const int seq = a.row_seq[row0], pos0 = a.row_pos[row0], len = pos0 + rows;
    const PageList list = visible_pages<true>(a, pos0, len - 1);
    const int pps = (list.n + a.nsplit - 1) / a.nsplit, p0 = split * pps, np = max(0, min(list.n, p0 + pps) - p0);
    const int32_t* pt = a.pool.page_table + (size_t)seq * a.pool.max_pages;
    for (int i = tid; i < np; i += B_THREADS) pt_s[i] = pt[list.page(p0 + i)];
    for (int e = warp; e < H; e += B_THREADS / 32)
        for (int h = lane; h < HP; h += 32) tk[e * HP + h] = h < H ? __ldg(a.talk + (size_t)h * H + e) : 0.f;
    for (int i = tid; i < pairs; i += B_THREADS) {
        const int r = i / H, h = i - r * H, g = h / gq, q = r * gq + h - g * gq;
        qi[i] = (uint16_t)(g * geo.per + q);
        if (g == 0) pair[q] = (uint16_t)i;
        ml[2 * i] = -INFINITY;
        ml[2 * i + 1] = 0.f;
    }
    const int o_tile = geo.cols2 * 8, o_n = G * vt_n * geo.ntile * o_tile;
    for (int i = tid; i < o_n; i += B_THREADS) os[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    __syncthreads();
    const unsigned char *kpool = reinterpret_cast<const unsigned char*>(a.pool.k), *vpool = reinterpret_cast<const unsigned char*>(a.pool.v);
    const uint32_t k_bytes = (uint32_t)(GQA_PAGE * dp * 2), v_bytes = (uint32_t)(GQA_PAGE * vp * 2);
    if (warp == ATT_WARPS) {
        if (lane == 0) {
            // blocks in order: a page's keys of every key head, then its values
            int s = 0, filled = 0;
            uint32_t phase = 1;  // of the stage's empty barrier; its first round needs no wait
            bool ok = true, waited = false;
            for (int i = 0; i < np && ok; ++i) {
                const size_t tile = (size_t)pt_s[i] * G;
                const bool settled = a.early && list.page(p0 + i) < (len - 1) / GQA_PAGE;  // complete before the launch in front began
                for (int b = 0; b < 2 * G; ++b) {
                    if (!waited && (!settled || filled == NST)) {
                        pdl_wait();
                        waited = true;
                    }
                    if (filled == NST && !mb_wait(&empty[s], phase, a.err_flag, &s_abort)) {
                        ok = false;
                        break;
                    }
                    const bool is_v = b >= G;
                    mb_expect_tx(&full[s], is_v ? v_bytes : k_bytes);
                    bulk_copy(ring + (size_t)s * geo.block, is_v ? vpool + (tile + b - G) * v_bytes : kpool + (tile + b) * k_bytes, is_v ? v_bytes : k_bytes, &full[s]);
                    if (filled < NST) ++filled;
                    if (++s == NST) {
                        s = 0;
                        phase ^= 1;
                    }
                }
            }
            if (!waited) pdl_wait();
        } else {
            pdl_wait();
        }
    } else {
        pdl_wait();
        // queries: three bf16 terms, a warp per (row, head)
#pragma unroll 2
        for (int p = warp; p < pairs; p += ATT_WARPS) {
            const float* q = a.q + (size_t)row0 * H * dim + (size_t)p * dim;
            uint16_t* dst = qs + (size_t)qi[p] * ldq;
#pragma unroll 2
            for (int d = 2 * lane; d < dp; d += 64) {
                float x = 0.f, y = 0.f;
                if ((dim & 1) == 0) {
                    if (d < dim) {
                        const float2 v = __ldcg(reinterpret_cast<const float2*>(q + d));
                        x = v.x;
                        y = v.y;
                    }
                } else {
                    x = d < dim ? __ldcg(q + d) : 0.f;
                    y = d + 1 < dim ? __ldcg(q + d + 1) : 0.f;
                }
                uint32_t t[3];
                bf16x2_split3(x, y, t[0], t[1], t[2]);
#pragma unroll
                for (int k = 0; k < 3; ++k) *reinterpret_cast<uint32_t*>(dst + (size_t)k * padded * ldq + d) = t[k];
            }
        }
        asm volatile("bar.sync 1, 256;" ::: "memory");
        const int gid = lane >> 2, tig = lane & 3, mj = lane >> 3, mr = lane & 7, valid = rows * gq;
        const uint32_t k_lane = (uint32_t)(((mj >> 1) * GQA_PAGE + (mj & 1) * 8 + mr) * 16), v_lane = (uint32_t)(((mj & 1) * GQA_PAGE + (mj >> 1) * 8 + mr) * 16);
        const int kh = pairs > 16 ? 4 : pairs > 8 ? 2 : 1, hu = (H + kh - 1) / kh;  // heads of a unit of the mixing: few enough that every warp has one
        const uint16_t *q_lane = qs + (size_t)gid * ldq + 2 * tig, *p_lane = ps + (size_t)gid * TALK_P_LD + 2 * tig;
        const bool kept = tig < geo.cols2;
        int s = 0;
        uint32_t phase = 0;
        auto next = [&]() {
            __syncwarp();
            if (lane == 0) mb_arrive(&empty[s]);
            if (++s == NST) {
                s = 0;
                phase ^= 1;
            }
        };
        for (int i = 0; i < np; ++i) {
            const int tok0 = list.page(p0 + i) * GQA_PAGE;
            // scores.  A wait that gives up leaves the work out; the barriers below are still met by every warp.
            for (int g = 0; g < G; ++g) {
                const bool ok = __all_sync(0xffffffffu, mb_wait(&full[s], phase, a.err_flag, &s_abort));
                const uint32_t kb = s32(ring + (size_t)s * geo.block) + k_lane;
                for (int j = (warp - g * 4 * geo.ntile) & 7; ok && j < 4 * geo.ntile; j += 8) {
                    const int u = j & 3, nt = j >> 2;
                    float sc[3][4];
#pragma unroll
                    for (int k = 0; k < 3; ++k) sc[k][0] = sc[k][1] = sc[k][2] = sc[k][3] = 0.f;
                    const uint16_t* q = q_lane + (size_t)(g * geo.per + nt * 8) * ldq;
                    const uint32_t ku = kb + (uint32_t)(u * 256);
#pragma unroll 4
                    for (int kt = 0; kt < kt_n; ++kt) {
                        uint32_t ka[4];
                        ldsm4(ka, ku + (uint32_t)(kt * (2 * GQA_PAGE * 16)));
#pragma unroll
                        for (int k = 0; k < 3; ++k) {
                            const uint16_t* b = q + (size_t)k * padded * ldq + kt * 16;
                            mma16816(sc[k], ka, *reinterpret_cast<const uint32_t*>(b), *reinterpret_cast<const uint32_t*>(b + 8));
                        }
                    }
#pragma unroll
                    for (int hh = 0; hh < 2; ++hh) {
                        const int c = nt * 8 + 2 * tig + hh;
                        if (c < valid) {
                            float* dst = raw + (size_t)(pair[c] + g * gq) * TALK_RAW_LD + u * 16 + gid;
                            dst[0] = (sc[2][hh] + sc[1][hh]) + sc[0][hh];
                            dst[8] = (sc[2][2 + hh] + sc[1][2 + hh]) + sc[0][2 + hh];
                        }
                    }
                }
                next();
            }
            asm volatile("bar.sync 1, 256;" ::: "memory");
            for (int w = warp; w < rows * hu; w += ATT_WARPS) {
                const int r = rows == 1 ? 0 : w / hu, h0 = (w - r * hu) * kh, pos = pos0 + r, from = first_visible(a, pos), ta = tok0 + 2 * lane;
                const float* x = raw + (size_t)r * H * TALK_RAW_LD + 2 * lane;
                if (kh == 4) talk_mix<4>(a, r, h0, pos, from, ta, x, tk, HP, qi, ps, padded, ml, corr);
                else if (kh == 2) talk_mix<2>(a, r, h0, pos, from, ta, x, tk, HP, qi, ps, padded, ml, corr);
                else talk_mix<1>(a, r, h0, pos, from, ta, x, tk, HP, qi, ps, padded, ml, corr);
            }
            asm volatile("bar.sync 1, 256;" ::: "memory");
            for (int g = 0; g < G; ++g) {
                const bool ok = __all_sync(0xffffffffu, mb_wait(&full[s], phase, a.err_flag, &s_abort));
                const uint32_t vb = s32(ring + (size_t)s * geo.block) + v_lane;
                const int units = vt_n * geo.ntile;
                for (int j = (warp - g * units) & 7; ok && j < units; j += 8) {
                    const int nt = geo.ntile == 1 ? 0 : j / vt_n, mt = j - nt * vt_n, q0 = g * geo.per + nt * 8;
                    float4* o = os + (size_t)((g * vt_n + mt) * geo.ntile + nt) * o_tile + tig * 8 + gid;
                    const float4 c = kept ? *o : make_float4(0.f, 0.f, 0.f, 0.f);
                    const float c0 = corr[q0 + 2 * tig], c1 = corr[q0 + 2 * tig + 1];
                    float acc[3][4] = {{c.x * c0, c.y * c1, c.z * c0, c.w * c1}, {0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
                    const uint16_t* p = p_lane + (size_t)q0 * TALK_P_LD;
#pragma unroll
                    for (int kt = 0; kt < 4; ++kt) {
                        uint32_t va[4];
                        ldsm4_trans(va, vb + (uint32_t)(mt * (2 * GQA_PAGE * 16) + kt * 256));
#pragma unroll
                        for (int k = 0; k < 3; ++k) {
                            const uint16_t* b = p + (size_t)k * padded * TALK_P_LD + kt * 16;
                            mma16816(acc[k], va, *reinterpret_cast<const uint32_t*>(b), *reinterpret_cast<const uint32_t*>(b + 8));
                        }
                    }
                    if (kept) *o = make_float4((acc[2][0] + acc[1][0]) + acc[0][0], (acc[2][1] + acc[1][1]) + acc[0][1], (acc[2][2] + acc[1][2]) + acc[0][2], (acc[2][3] + acc[1][3]) + acc[0][3]);
                }
                next();
            }
        }
    }
    __syncthreads();  // every block consumed: the ring takes the results
    float* res = reinterpret_cast<float*>(ring);  // [row][head][ldo]
    {
        const int gid = lane & 7, tig = lane >> 3;
        for (int gm = warp; gm < G * vt_n; gm += B_THREADS / 32) {
            const int g = gm / vt_n, mt = gm - g * vt_n;
            for (int nt = 0; nt < geo.ntile; ++nt) {
                if (tig >= geo.cols2) continue;
                const float4 v = os[(size_t)(gm * geo.ntile + nt) * o_tile + lane];
                const float x[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
                for (int k = 0; k < 2; ++k) {
                    const int c = nt * 8 + 2 * tig + k;
                    if (c >= rows * gq) continue;
                    float* d = res + (size_t)(pair[c] + g * gq) * ldo + mt * 16 + gid;
                    d[0] = x[k];
                    d[8] = x[2 + k];
                }
            }
        }
    }
    __syncthreads();
    auto store = [&](int p, int d0, float (&v)[8]) {
        const int r = rows == 1 ? 0 : p / H;
        store_piece<true>(a, row0 + r, p - r * H, d0, v);
    };
    const int np8 = vp / 8, np4 = vp / 4;
    if (ns == 1) {
        for (int i = tid; i < pairs * np8; i += B_THREADS) {
            const int p = i / np8, d0 = (i - p * np8) * 8;
            const float4 x = *reinterpret_cast<const float4*>(res + (size_t)p * ldo + d0), y = *reinterpret_cast<const float4*>(res + (size_t)p * ldo + d0 + 4);
            const int h = rows == 1 ? p : p % H;
            const float f = 1.0f / (ml[2 * p + 1] + sink_weight<true>(a, h, ml[2 * p]));
            float v[8] = {x.x * f, x.y * f, x.z * f, x.w * f, y.x * f, y.y * f, y.z * f, y.w * f};
            if (d0 < vdim) store(p, d0, v);
        }
        return;
    }
    for (int i = tid; i < pairs * np4; i += B_THREADS) {
        const int p = i / np4, d = (i - p * np4) * 4, k = p / ns;
        const uint32_t owner = (uint32_t)(p - k * ns);
        const float4 v = *reinterpret_cast<const float4*>(res + (size_t)p * ldo + d);
        float* slot = recv + (size_t)(rank * own_most + k) * (vp + 4);
        if ((int)owner == rank) {
            *reinterpret_cast<float4*>(slot + d) = v;
            if (d == 0) {
                slot[vp] = ml[2 * p];
                slot[vp + 1] = ml[2 * p + 1];
            }
        } else {
            const uint32_t bar = dsmem_addr(&s_rbar, owner);
            st_async_f32x4(dsmem_addr(slot + d, owner), v, bar);
            if (d == 0) st_async_f32x2(dsmem_addr(slot + vp, owner), ml[2 * p], ml[2 * p + 1], bar);
        }
    }
    if (own == 0) return;
    __syncthreads();
    if (!mb_wait_cluster(&s_rbar, 0, a.err_flag, &s_abort)) return;  // bounded
    for (int i = tid; i < own * np8; i += B_THREADS) {
        const int k = i / np8, d0 = (i - k * np8) * 8, p = k * ns + rank;
        float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f}, mx = -INFINITY, l = 0.f;
        for (int r = 0; r < ns; ++r) mx = fmaxf(mx, recv[(size_t)(r * own_most + k) * (vp + 4) + vp]);
#pragma unroll 4
        for (int r = 0; r < ns; ++r) {
            const float* slot = recv + (size_t)(r * own_most + k) * (vp + 4);
            const float f = slot[vp] == -INFINITY ? 0.f : exp2f(slot[vp] - mx);
            const float4 x = *reinterpret_cast<const float4*>(slot + d0), y = *reinterpret_cast<const float4*>(slot + d0 + 4);
            l = fmaf(f, slot[vp + 1], l);
            v[0] = fmaf(f, x.x, v[0]); v[1] = fmaf(f, x.y, v[1]); v[2] = fmaf(f, x.z, v[2]); v[3] = fmaf(f, x.w, v[3]);
            v[4] = fmaf(f, y.x, v[4]); v[5] = fmaf(f, y.y, v[5]); v[6] = fmaf(f, y.z, v[6]); v[7] = fmaf(f, y.w, v[7]);
        }
        const float inv = 1.0f / (l + sink_weight<true>(a, rows == 1 ? p : p % H, mx));
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] *= inv;
        if (d0 < vdim) store(p, d0, v);
    }
}

inline size_t talk_plain_smem(int heads, int dp, int vp, int nsplit) { return sizeof(float) * (size_t)heads * (dp + vp + 4 + 2 * GQA_PAGE + 3 + nsplit); }

inline cudaError_t launch_talk(GqaAttnArgs a, int sm_count, cudaStream_t st, bool pdl) {
    const int dp = gqa_pad(a.pool.dim), vp = gqa_pad(a.pool.vdim);
    TalkGeom g{};
    auto pages_of = [&](int rows) { return most_pages(a, rows * a.heads / a.pool.kv_heads); };
    if (a.pool.bf16 && pages_of(1) <= 4096) {
        const int gq = a.heads / a.pool.kv_heads;
        const int asked = a.nsplit;
        // rows of a run share a tile until the columns of an MMA are full
        for (int rows = std::max(1, std::min(8 / gq, a.longest_run)); rows >= 1; rows /= 2) {
            const int pages = pages_of(rows);
            a.tiles = a.M;
            if (a.runs.n > 0) {
                a.tiles = 0;
                for (int r = 0; r < a.runs.n; ++r) {
                    a.runs.tile[r] = (uint16_t)a.tiles;
                    a.tiles += (a.runs.row[r + 1] - a.runs.row[r] + rows - 1) / rows;
                }
                a.runs.tile[a.runs.n] = (uint16_t)a.tiles;
            }
            // first as many splits as keep two CTAs on every SM, which hide one another's barriers, then one with a deep ring
            bool fits = false;
            for (int per_sm = pages > 2 ? 2 : 1; per_sm >= 1 && !fits; --per_sm) {
                const size_t most = (per_sm == 2 ? 112 : 226) * 1024;
                auto shape = [&](int n) {
                    a.nsplit = n;
                    return talk_geom(a, rows, n, (pages + n - 1) / n, most, &g) && (per_sm == 1 || g.stages >= 4);
                };
                if (asked > 0) {
                    fits = shape(asked);
                    continue;
                }
                for (int n = std::max(1, std::min({per_sm * sm_count / a.tiles, a.max_cluster, 8, pages})); n >= 1 && !fits; --n)
                    fits = shape(n) && (n == 1 || clusters_at_once(talk_attn_mma_kernel, n, B_THREADS, g.smem) >= a.tiles);
            }
            if (fits) return launch_clustered(talk_attn_mma_kernel, dim3((unsigned)a.nsplit, 1, (unsigned)a.tiles), dim3(B_THREADS), g.smem, a.nsplit, st, pdl, a, g);
        }
        a.nsplit = asked;
    }
    const int pages = most_pages(a, 1);
    if (a.nsplit < 1) a.nsplit = std::max(1, std::min({2 * sm_count / a.M, a.max_cluster, 8, pages}));
    const size_t smem = talk_plain_smem(a.heads, dp, vp, a.nsplit);
    if (smem > 226 * 1024) return cudaErrorInvalidValue;
    const dim3 grid((unsigned)a.nsplit, 1, (unsigned)a.M);
    return a.pool.bf16 ? launch_clustered(gqa_attn_kernel<true, true, true>, grid, dim3(A_THREADS), smem, a.nsplit, st, pdl, a)
                       : launch_clustered(gqa_attn_kernel<false, true, true>, grid, dim3(A_THREADS), smem, a.nsplit, st, pdl, a);
}
