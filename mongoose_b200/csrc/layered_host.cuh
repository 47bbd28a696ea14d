// Host side of layer-described models: buffers, weights, one token (a captured sequence of phase kernels,
// like enqueue_step's) and portions of a prompt.  Included by engine.cu, whose engine, arena, cursor,
// graph cache and stepping calls it shares.
#pragma once

struct LayerWeights {
    mg_layer_config c{};
    uint8_t* proj = nullptr;            // the mixer's input matrices, stacked
    float *norm1 = nullptr, *norm2 = nullptr;
    // MG_MIXER_PARALLEL
    ProjCols cols{};
    int splits = 1, tile = 16;
    int block_rows = 0;                 // queries per block of the tensor-core attention; 0: CUDA-core kernel
    uint8_t *at_o = nullptr, *mem_o = nullptr, *up = nullptr, *down = nullptr;
    float *at_out = nullptr, *mem_out = nullptr;
    float *q_norm = nullptr, *k_norm = nullptr, *talk = nullptr, *bias = nullptr, *slopes = nullptr;
    float *mem_norm = nullptr, *i_bias = nullptr, *f_bias = nullptr;
    GateAttn at{};
    MatMem mem{};
    // the other mixers: `o` is their output matrix
    float *ls1 = nullptr, *ls2 = nullptr;
    uint8_t *o = nullptr, *uq = nullptr, *uk = nullptr, *uv = nullptr, *w2 = nullptr;
    float *dq_norm = nullptr, *dkv_norm = nullptr, *cos_tab = nullptr, *sin_tab = nullptr;
    float *mu[5] = {}, *w0 = nullptr, *u = nullptr, *wkv_norm = nullptr;
    LatentAttn la{};
    Wkv wk{};
    int group = 1;                      // heads per CTA of the attention over cached rows
    bool latent_tc = false;
    // mixture of experts: `router` is the router, the shared expert's gate, its gate and its up projection
    uint8_t *router = nullptr, *e_gate = nullptr, *e_up = nullptr, *e_down = nullptr, *shared_down = nullptr;
    float* moe_bias = nullptr;
    Moe moe{};

    bool parallel() const { return c.mixer == MG_MIXER_PARALLEL; }
    int kat() const { return c.attn.heads * c.attn.dim; }
    int kmem() const { return c.mem.heads * c.mem.vdim; }
    int kout() const { return c.mixer == MG_MIXER_LATENT ? c.latent.heads * c.latent.vdim : c.wkv.heads * c.wkv.dim; }
    int proj_rows() const {
        return parallel() ? cols.total : c.mixer == MG_MIXER_LATENT ? c.latent.q_rank + c.latent.kv_rank + c.latent.rot_dim : 4 * kout() + c.wkv.decay_rank;
    }
    int router_rows() const { return moe.experts + (moe.shared_ff ? 1 + 2 * moe.shared_ff : 0); }
    uint8_t* router_row(int r) const { return router + (size_t)r * moe.ldw * 2; }
};

// One run of a layer: a looped layer has several, each with its own cache or state.
struct LayerRun {
    int layer = 0;
    bool begins = false;                // a pass of the loop begins here
    void* cache = nullptr;              // keys, or latents and rotated key parts
    float *cache_r = nullptr, *S = nullptr, *nrm = nullptr, *mx = nullptr;
    float* prev = nullptr;              // [2][width] the last token's normed vector, by the parity of the position
    int next_pos = 0;                   // tokens this run's cache and state have seen
    GateAttn at(const LayerWeights& l) const { GateAttn a = l.at; a.cache = cache; a.cache_r = cache_r; return a; }
    MatMem mem(const LayerWeights& l) const { MatMem a = l.mem; a.S = S; a.nrm = nrm; a.m = mx; return a; }
    LatentAttn la(const LayerWeights& l) const { LatentAttn a = l.la; a.cache = cache; return a; }
    Wkv wk(const LayerWeights& l) const { Wkv a = l.wk; a.S = S; return a; }
};

struct LayerSlot {
    int rows = 0, cols = 0;             // 0: the slot does not exist
    uint8_t* mat = nullptr;             // bf16 rows padded to pad_to(cols, 64)
    std::vector<int> place;             // row of the matrix -> row in memory, where heads are padded
    int place_rows = 0;
    float* vec = nullptr;
    bool rounds = false;                // a small matrix among the vectors: held as fp32, rounded to bf16
    bool set = false;
};

struct Layered {
    mg_model_config c{};
    bool f32 = false;
    int kw = 0;                         // padded width
    int kl = 0;                         // padded row length of the loop's input matrix
    std::vector<LayerWeights> layers;
    std::vector<LayerRun> runs;
    std::vector<LayerSlot> slots;
    uint8_t *embed = nullptr, *head = nullptr, *loop_in = nullptr;
    float *final_norm = nullptr, *pos_tab = nullptr;
    // one token
    float *row = nullptr, *part = nullptr, *attn = nullptr, *mem_raw = nullptr, *mem_y = nullptr, *y[2] = {}, *z = nullptr, *mid = nullptr;
    float *x0 = nullptr, *hn = nullptr, *q1 = nullptr, *rt = nullptr, *emid = nullptr;
    int* esel = nullptr;
    float *qa = nullptr, *lpart = nullptr;      // latent attention: folded queries, partial sums (one token, or all rows)
    float2* ml = nullptr;
    // portions
    int max_rows = 0, logit_rows = 0;
    int *tokens = nullptr, *want = nullptr;
    float *x = nullptr, *P = nullptr, *yr[2] = {}, *zr = nullptr, *logits = nullptr;
    uint8_t *act = nullptr, *qh = nullptr, *ao = nullptr, *my = nullptr, *midr = nullptr, *fin = nullptr;
    uint8_t *aw = nullptr, *vt = nullptr;   // tensor-core attention: mixed weights of a query block, transposed keys or values
    uint8_t* keys = nullptr;            // keys formed from latents
    float *x0r = nullptr, *hr = nullptr, *q32 = nullptr, *decay = nullptr, *wo = nullptr, *rtr = nullptr, *glu = nullptr, *inner32 = nullptr;
    uint8_t *cat = nullptr, *mix = nullptr, *inner = nullptr, *cq = nullptr, *xmid = nullptr;
    MoeRows moe{};
    MemRows mw{};
    int np = 0;                         // widest projection row
    int* status = nullptr;              // set by a wait inside a tensor-core kernel that ran out
};

namespace {

constexpr int kThinSlices = 8;      // slices of layered_matmul_thin, at most

// Runs `take(pointer, bytes)` over every device buffer of the model, so that sizing the arena and
// carving it are one list.
template <typename F>
int layered_buffers(Layered& m, F take) {
    const mg_model_config& c = m.c;
    const int W = c.width, kw = m.kw, T = m.max_rows, ldv = pad_to(c.max_seq, 64);
    const size_t as = m.f32 ? 4 : 2;
    int rc = 0;
    auto get = [&](auto** p, size_t count, size_t elem) {
        if (!rc && count) rc = take((void**)p, count * elem);
    };
    size_t hd = 0, kat = 1, kmem = 0, ff = 0, mh = 0, u = 0, nu = 0, part = 0, aw = 0, vt = 0;
    size_t q1 = 0, q32 = 0, qa = 0, lpart = 0, ml = 0, keys = 0, cq = 0, wkv = 0, ld2 = 0, rt = 0, rtr = 0, emid = 0, xmid = 0, moe = 0, tiles = 0, top = 0, experts = 0;
    bool any_post = false, any_pre = false;
    for (size_t i = 0; i < m.layers.size(); i++) {
        LayerWeights& l = m.layers[i];
        get(&l.proj, (size_t)l.proj_rows() * kw, 2);
        get(&l.norm1, W, 4);
        if (l.parallel()) {
            const mg_gate_attn_config& a = l.c.attn;
            const mg_mat_mem_config& r = l.c.mem;
            any_post = true;
            get(&l.at_o, (size_t)W * pad_to(l.kat(), 64), 2);
            get(&l.mem_o, (size_t)W * pad_to(l.kmem(), 64), 2);
            get(&l.at_out, W, 4); get(&l.mem_out, W, 4);
            if (l.c.ffn_dim) {
                get(&l.norm2, W, 4);
                get(&l.up, (size_t)l.c.ffn_dim * kw, 2);
                get(&l.down, (size_t)W * pad_to(l.c.ffn_dim, 64), 2);
            }
            get(&l.q_norm, a.dim, 4); get(&l.k_norm, a.dim, 4); get(&l.talk, (size_t)a.heads * a.heads, 4);
            get(&l.bias, a.heads, 4); get(&l.slopes, a.heads, 4);
            get(&l.mem_norm, l.kmem(), 4); get(&l.i_bias, r.heads, 4); get(&l.f_bias, r.heads, 4);
            hd = std::max(hd, (size_t)a.heads * l.at.dim_s);
            kat = std::max(kat, (size_t)pad_to(l.kat(), 64)); kmem = std::max(kmem, (size_t)pad_to(l.kmem(), 64));
            ff = std::max(ff, (size_t)pad_to(l.c.ffn_dim, 64)); mh = std::max(mh, (size_t)r.heads);
            const size_t chunks = (T + kMemChunk - 1) / kMemChunk;
            u = std::max(u, chunks * r.heads * r.dim * r.vdim); nu = std::max(nu, chunks * r.heads * r.dim);
            if (l.block_rows) {
                aw = std::max(aw, (size_t)a.heads * l.block_rows * ldv);
                vt = std::max(vt, (size_t)a.kv_heads * a.dim * ldv);
            }
            part = std::max(part, (size_t)l.splits * a.heads * l.at.dim_s);
            continue;
        }
        any_pre = true;
        get(&l.ls1, W, 4);
        get(&l.o, (size_t)W * pad_to(l.kout(), 64), 2);
        kat = std::max(kat, (size_t)pad_to(l.kout(), 64));
        if (l.c.mixer == MG_MIXER_LATENT) {
            const LatentAttn& a = l.la;
            get(&l.dq_norm, a.q_rank, 4); get(&l.dkv_norm, a.rank, 4);
            get(&l.uq, (size_t)a.heads * a.qrow() * pad_to(a.q_rank, 64), 2);
            get(&l.uk, (size_t)a.heads * a.dim_s * a.ld, 2); get(&l.uv, (size_t)a.heads * a.vdim * a.ld, 2);
            const LayerWeights* like = nullptr;         // an earlier layer with the same rotation
            for (size_t k = 0; k < i && !like; k++)
                if (m.layers[k].c.mixer == MG_MIXER_LATENT && m.layers[k].c.latent.rot_dim == a.rot && m.layers[k].c.latent.rot_base == l.c.latent.rot_base)
                    like = &m.layers[k];
            if (like) { l.cos_tab = like->cos_tab; l.sin_tab = like->sin_tab; }
            else { get(&l.cos_tab, (size_t)c.max_seq * (a.rot / 2), 4); get(&l.sin_tab, (size_t)c.max_seq * (a.rot / 2), 4); }
            q1 = std::max(q1, (size_t)a.heads * a.qrow());
            q32 = std::max(q32, (size_t)T * a.heads * a.qrow());
            // rows that do not go through the tensor cores: every token like the one of a decode step, one range each
            const size_t rows = l.latent_tc ? 1 : T;
            qa = std::max(qa, rows * a.heads * a.row());
            const size_t ranges = std::max((size_t)l.splits, rows);
            lpart = std::max(lpart, ranges * a.heads * a.rank_s); ml = std::max(ml, ranges * a.heads);
            if (l.latent_tc) {
                hd = std::max(hd, (size_t)a.heads * a.qrow());
                keys = std::max(keys, (size_t)c.max_seq * a.heads * a.dim_s);
                vt = std::max(vt, (size_t)a.heads * a.vdim * ldv);
            }
            cq = std::max(cq, (size_t)pad_to(a.q_rank, 64));
        } else {
            const int n = l.kout();
            for (float*& v : l.mu) get(&v, W, 4);
            get(&l.w2, (size_t)n * l.wk.ld2, 2);
            get(&l.w0, n, 4); get(&l.u, n, 4); get(&l.wkv_norm, n, 4);
            wkv = std::max(wkv, (size_t)n); ld2 = std::max(ld2, (size_t)2 * l.wk.ld2);
        }
        if (l.moe.experts) {
            const Moe& e = l.moe;
            get(&l.norm2, W, 4); get(&l.ls2, W, 4); get(&l.moe_bias, e.experts, 4);
            get(&l.router, (size_t)l.router_rows() * kw, 2);
            get(&l.e_gate, (size_t)e.experts * e.ff * kw, 2); get(&l.e_up, (size_t)e.experts * e.ff * kw, 2);
            get(&l.e_down, (size_t)e.experts * W * e.ffs, 2);
            get(&l.shared_down, (size_t)(e.shared_ff ? W : 0) * e.shared_ffs, 2);
            const size_t nt = moe_tiles(e, T), rows = nt * 128;
            rt = std::max(rt, (size_t)l.router_rows()); rtr = std::max(rtr, (size_t)pad_to(e.experts + 1, 4));
            emid = std::max(emid, (size_t)e.top * e.ffs + e.shared_ffs);
            xmid = std::max(xmid, std::max(rows * e.ffs, (size_t)T * e.shared_ffs));
            moe = std::max(moe, rows); tiles = std::max(tiles, nt); top = std::max(top, (size_t)e.top); experts = std::max(experts, (size_t)e.experts);
        }
    }
    for (LayerRun& r : m.runs) {
        const LayerWeights& l = m.layers[r.layer];
        if (l.parallel()) {
            get(&r.cache, (size_t)c.max_seq * l.at.kv_heads * l.at.dim_s, as);
            get(&r.cache_r, (size_t)c.max_seq * l.at.kv_heads, 4);
            get(&r.S, (size_t)l.mem.heads * l.mem.dim * l.mem.vdim, 4);
            get(&r.nrm, (size_t)2 * l.mem.heads * l.mem.dim, 4);
            get(&r.mx, (size_t)2 * l.mem.heads, 4);
        } else if (l.c.mixer == MG_MIXER_LATENT) {
            get(&r.cache, (size_t)c.max_seq * l.la.row(), as);
        } else {
            get(&r.S, (size_t)l.wk.heads * l.wk.dim * l.wk.dim, 4);
            get(&r.prev, (size_t)2 * W, 4);
        }
    }
    get(&m.embed, (size_t)c.vocab * kw, 2); get(&m.head, (size_t)c.vocab * kw, 2);
    if (c.loop_times) { get(&m.loop_in, (size_t)W * m.kl, 2); get(&m.x0, W, 4); get(&m.x0r, (size_t)T * W, 4); get(&m.cat, (size_t)T * m.kl, as); }
    get(&m.final_norm, W, 4);
    if (c.positions == MG_POS_SINUSOID) get(&m.pos_tab, (size_t)c.max_seq * W, 4);
    get(&m.row, m.np, 4); get(&m.part, part, 4); get(&m.attn, kat, 4);
    get(&m.mem_raw, kmem, 4); get(&m.mem_y, kmem, 4); get(&m.y[0], W, 4); get(&m.y[1], W, 4); get(&m.z, W, 4); get(&m.mid, ff, 4);
    get(&m.hn, any_pre ? kw : 0, 4); get(&m.q1, q1, 4); get(&m.rt, rt, 4); get(&m.emid, emid, 4);
    get(&m.qa, qa, 4); get(&m.lpart, lpart, 4); get(&m.ml, ml, 8);
    get(&m.status, 1, 4); get(&m.tokens, T, 4); get(&m.want, T, 4);
    get(&m.x, (size_t)T * W, 4); get(&m.P, (size_t)T * m.np, 4);
    for (float*& y : m.yr) get(&y, any_post ? (size_t)T * W : 0, 4);
    get(&m.zr, (size_t)T * W, 4);
    get(&m.logits, (size_t)m.logit_rows * c.vocab, 4);
    get(&m.act, (size_t)T * kw, as); get(&m.qh, (size_t)T * hd, as); get(&m.ao, (size_t)T * kat, as);
    get(&m.my, (size_t)T * kmem, as); get(&m.midr, (size_t)T * ff, as); get(&m.fin, (size_t)m.logit_rows * kw, as);
    get(&m.aw, aw, 2); get(&m.vt, vt, 2); get(&m.keys, keys, 2);
    get(&m.q32, q32, 4); get(&m.cq, (size_t)T * cq, as);
    if (wkv) { get(&m.hr, (size_t)T * W, 4); get(&m.mix, (size_t)5 * T * kw, as); get(&m.decay, (size_t)T * wkv, 4); get(&m.wo, (size_t)T * wkv, 4); get(&m.inner, m.f32 ? 0 : (size_t)T * ld2, 2); get(&m.inner32, (size_t)kThinSlices * T * (ld2 / 2), 4); }
    get(&m.rtr, (size_t)kThinSlices * T * rtr, 4); get(&m.moe.shared_gate, rtr ? T : 0, 4); get(&m.xmid, xmid, as); get(&m.glu, m.f32 ? xmid : 0, 4);
    get(&m.moe.sel, (size_t)T * top, 4); get(&m.moe.slot, (size_t)T * top, 4); get(&m.moe.weight, (size_t)T * top, 4);
    get(&m.moe.count, experts, 4); get(&m.moe.first, experts ? experts + 1 : 0, 4); get(&m.moe.group, tiles, 4);
    get(&m.moe.x, moe * kw, as); get(&m.moe.y, moe * W, as);
    get(&m.esel, top, 4);
    get(&m.mw.b, (size_t)mh * T, 8); get(&m.mw.ig, (size_t)mh * T, 4); get(&m.mw.mm, (size_t)mh * T, 4); get(&m.mw.m0, mh, 4);
    get(&m.mw.g, (size_t)mh * ((T + kMemChunk - 1) / kMemChunk), 4);
    get(&m.mw.U, u, 4); get(&m.mw.nU, nu, 4); get(&m.mw.o, (size_t)T * kmem, 4);
    return rc;
}

// Shapes and kernel arguments of one layer.
int parallel_shapes(Layered& m, LayerWeights& l, int sms, std::string* why) {
    const mg_model_config& c = m.c;
    const mg_gate_attn_config& a = l.c.attn;
    const mg_mat_mem_config& r = l.c.mem;
    if (a.heads <= 0 || a.kv_heads <= 0 || a.heads % a.kv_heads || a.dim <= 0 || a.temp_every <= 0 ||
        r.heads <= 0 || r.dim <= 0 || r.vdim <= 0 || !(r.gate_cap > 0.f) || l.c.ffn_dim < 0) { *why = "bad layer sizes"; return MG_ERR_ARG; }
    GateAttn& g = l.at;
    g.heads = a.heads; g.kv_heads = a.kv_heads; g.dim = a.dim; g.dim_s = pad_to(a.dim, 8);
    g.scale = a.scale; g.temp_coef = a.temp_coef; g.temp_every = a.temp_every; g.eps = c.norm_eps; g.max_seq = c.max_seq;
    MatMem& q = l.mem;
    q.heads = r.heads; q.dim = r.dim; q.vdim = r.vdim; q.cap = r.gate_cap; q.eps = c.norm_eps;
    const int n_mem = r.heads * ((r.vdim + 31) / 32);
    l.splits = std::max(32, sms - n_mem);
    if (!mixer_step_smem(g, q, m.f32, &l.tile)) { *why = "attention heads do not fit one CTA's registers or shared memory"; return MG_ERR_UNSUPPORTED; }
    if (!m.f32 && gate_attn_tc_fits(g)) l.block_rows = gate_attn_tc_rows(g, c.max_seq, m.max_rows, (size_t)256 << 20);
    ProjCols& p = l.cols;
    int o = 0;
    auto col = [&](int n) { const int at = o; o += n; return at; };
    p.q = col(a.heads * a.dim); p.k = col(a.kv_heads * a.dim);
    p.mq = col(r.heads * r.dim); p.mk = col(r.heads * r.dim); p.mv = col(r.heads * r.vdim); p.mg = col(r.heads * r.vdim);
    p.mi = col(r.heads); p.mf = col(r.heads);
    p.total = o;
    return MG_OK;
}

int prenorm_shapes(Layered& m, LayerWeights& l, int sms, std::string* why) {
    const mg_model_config& c = m.c;
    if (l.c.mixer == MG_MIXER_LATENT) {
        const mg_latent_attn_config& a = l.c.latent;
        if (a.heads <= 0 || a.dim <= 0 || a.rot_dim <= 0 || a.rot_dim % 2 || a.vdim <= 0 || a.q_rank <= 0 || a.kv_rank <= 0 ||
            !(a.rot_base > 0.0)) { *why = "bad latent attention sizes"; return MG_ERR_ARG; }
        LatentAttn& g = l.la;
        g.heads = a.heads; g.dim = a.dim; g.rot = a.rot_dim; g.vdim = a.vdim; g.rank = a.kv_rank; g.q_rank = a.q_rank;
        g.dim_s = pad_to(a.dim, 8); g.rot_s = pad_to(a.rot_dim, 8); g.rank_s = pad_to(a.kv_rank, 8); g.ld = pad_to(a.kv_rank, 64);
        g.scale = a.scale; g.eps = c.norm_eps; g.max_seq = c.max_seq;
        if (!latent_attend_smem(g, m.f32, &l.tile, &l.group)) { *why = "a cached latent does not fit one CTA's registers or shared memory"; return MG_ERR_UNSUPPORTED; }
        l.splits = std::max(1, sms / ((a.heads + l.group - 1) / l.group));
        l.latent_tc = !m.f32 && latent_attn_tc_fits(g);
    } else {
        const mg_wkv_config& a = l.c.wkv;
        if (a.heads <= 0 || a.dim <= 0 || a.decay_rank <= 0) { *why = "bad recurrence sizes"; return MG_ERR_ARG; }
        Wkv& g = l.wk;
        g.heads = a.heads; g.dim = a.dim; g.rank = a.decay_rank; g.eps = c.norm_eps; g.ld2 = pad_to(a.decay_rank, 64);
        if (!wkv_rows_fits(g) || wkv_step_smem(g) > 48 * 1024) { *why = "a recurrent head does not fit one CTA"; return MG_ERR_UNSUPPORTED; }
    }
    const mg_moe_config& e = l.c.moe;
    if (!e.experts) return MG_OK;
    if (e.experts < 0 || e.top < 1 || e.top > e.experts || e.ff <= 0 || e.shared_ff < 0) { *why = "bad expert sizes"; return MG_ERR_ARG; }
    if (e.experts > kMaxExperts || e.top > kMaxTop) { *why = "more experts than the choice holds"; return MG_ERR_UNSUPPORTED; }
    Moe& g = l.moe;
    g.experts = e.experts; g.top = e.top; g.ff = e.ff; g.shared_ff = e.shared_ff; g.width = c.width;
    g.ffs = pad_to(e.ff, 64); g.shared_ffs = pad_to(e.shared_ff, 64); g.ldw = m.kw;
    const size_t smem = moe_step_smem(g);
    if (smem > 200 * 1024) { *why = "the chosen experts' inner vectors do not fit one CTA"; return MG_ERR_UNSUPPORTED; }
    return MG_OK;
}

// Shapes, runs and kernel arguments; MG_ERR_ARG / MG_ERR_UNSUPPORTED with a reason in *why.
int layered_shapes(Layered& m, int sms, std::string* why) {
    const mg_model_config& c = m.c;
    if (c.width <= 0 || c.vocab <= 0 || c.n_layers <= 0 || c.max_seq <= 0 || !(c.norm_eps >= 0.f) ||
        (c.math != MG_MATH_BF16 && c.math != MG_MATH_F32) || c.norm < MG_NORM_RMS_AROUND_ZERO || c.norm > MG_NORM_RMS ||
        (c.positions != MG_POS_SINUSOID && c.positions != MG_POS_NONE)) { *why = "bad model sizes"; return MG_ERR_ARG; }
    if (c.loop_times < 0 || (c.loop_times && (c.loop_start < 0 || c.loop_stop <= c.loop_start || c.loop_stop > c.n_layers))) { *why = "bad loop"; return MG_ERR_ARG; }
    m.f32 = c.math == MG_MATH_F32;
    m.kw = pad_to(c.width, 64);
    m.kl = pad_to(2 * c.width, 64);
    int kmax = std::max(m.kw, c.loop_times ? m.kl : 0);
    size_t moe_smem = 0;
    m.max_rows = std::min(c.max_seq, 2048);
    m.logit_rows = std::max(1, std::min(std::min(128, m.max_rows), (int)((64u << 20) / ((size_t)c.vocab * 4))));
    for (LayerWeights& l : m.layers) {
        if (l.c.mixer < MG_MIXER_PARALLEL || l.c.mixer > MG_MIXER_WKV) { *why = "unknown mixer"; return MG_ERR_ARG; }
        if (int rc = l.parallel() ? parallel_shapes(m, l, sms, why) : prenorm_shapes(m, l, sms, why)) return rc;
        m.np = std::max(m.np, pad_to(l.proj_rows(), 4));
        for (int k : {l.parallel() ? l.kat() : l.kout(), l.parallel() ? l.kmem() : 0, l.parallel() ? l.c.ffn_dim : 0, l.la.q_rank})
            kmax = std::max(kmax, pad_to(k, 64));
        if (l.moe.experts) moe_smem = std::max(moe_smem, moe_step_smem(l.moe));
    }
    for (int pass = 0, i = 0; i < c.n_layers;) {
        const bool looped = c.loop_times && i >= c.loop_start && i < c.loop_stop;
        LayerRun r;
        r.layer = i;
        r.begins = looped && i == c.loop_start;
        m.runs.push_back(r);
        i++;
        if (looped && i == c.loop_stop && ++pass < c.loop_times) i = c.loop_start;
    }
    // the phase kernels stage a whole input vector per CTA
    if (kmax > 48 * 1024) { *why = "a matrix with rows of more than 49152 values"; return MG_ERR_UNSUPPORTED; }
    if (layered_phase_smem(((size_t)kmax + 72) * sizeof(float)) != cudaSuccess) { *why = "kernel attributes"; return MG_ERR_CUDA; }
    if (moe_smem && moe_step_attrs(moe_smem) != cudaSuccess) { *why = "kernel attributes"; return MG_ERR_CUDA; }
    return MG_OK;
}

void layered_slots(Layered& m) {
    const mg_model_config& c = m.c;
    const int W = c.width;
    m.slots.assign((size_t)c.n_layers * MG_LAYER_SLOTS + 4, LayerSlot{});
    for (int i = 0; i < c.n_layers; i++) {
        LayerWeights& l = m.layers[i];
        LayerSlot* s = &m.slots[(size_t)i * MG_LAYER_SLOTS];
        auto vec = [&](int k, float* p, int n) { s[k].rows = 1; s[k].cols = n; s[k].vec = p; };
        auto mat = [&](int k, uint8_t* p, int row0, int rows, int cols) {
            s[k].rows = rows; s[k].cols = cols; s[k].mat = p + (size_t)row0 * pad_to(cols, 64) * 2;
        };
        vec(MG_SLOT_NORM1, l.norm1, W);
        if (l.parallel()) {
            const mg_gate_attn_config& a = l.c.attn;
            const mg_mat_mem_config& r = l.c.mem;
            mat(MG_SLOT_AT_Q, l.proj, l.cols.q, a.heads * a.dim, W); mat(MG_SLOT_AT_K, l.proj, l.cols.k, a.kv_heads * a.dim, W);
            vec(MG_SLOT_AT_QNORM, l.q_norm, a.dim); vec(MG_SLOT_AT_KNORM, l.k_norm, a.dim);
            vec(MG_SLOT_AT_TALK, l.talk, a.heads * a.heads); s[MG_SLOT_AT_TALK].rounds = true; vec(MG_SLOT_AT_BIAS, l.bias, a.heads);
            mat(MG_SLOT_AT_O, l.at_o, 0, W, l.kat()); vec(MG_SLOT_AT_OUT, l.at_out, W);
            mat(MG_SLOT_MEM_Q, l.proj, l.cols.mq, r.heads * r.dim, W); mat(MG_SLOT_MEM_K, l.proj, l.cols.mk, r.heads * r.dim, W);
            mat(MG_SLOT_MEM_V, l.proj, l.cols.mv, r.heads * r.vdim, W); mat(MG_SLOT_MEM_G, l.proj, l.cols.mg, r.heads * r.vdim, W);
            mat(MG_SLOT_MEM_O, l.mem_o, 0, W, l.kmem()); vec(MG_SLOT_MEM_NORM, l.mem_norm, l.kmem());
            mat(MG_SLOT_MEM_I, l.proj, l.cols.mi, r.heads, W); vec(MG_SLOT_MEM_IB, l.i_bias, r.heads);
            mat(MG_SLOT_MEM_F, l.proj, l.cols.mf, r.heads, W); vec(MG_SLOT_MEM_FB, l.f_bias, r.heads);
            vec(MG_SLOT_MEM_OUT, l.mem_out, W);
            if (l.c.ffn_dim) {
                vec(MG_SLOT_NORM2, l.norm2, W);
                mat(MG_SLOT_UP, l.up, 0, l.c.ffn_dim, W); mat(MG_SLOT_DOWN, l.down, 0, W, l.c.ffn_dim);
            }
            l.at.q_norm = l.q_norm; l.at.k_norm = l.k_norm; l.at.talk = l.talk; l.at.head_bias = l.bias; l.at.slopes = l.slopes;
            l.mem.i_bias = l.i_bias; l.mem.f_bias = l.f_bias; l.mem.norm = l.mem_norm;
            continue;
        }
        vec(MG_SLOT_LS1, l.ls1, W);
        if (l.c.mixer == MG_MIXER_LATENT) {
            LatentAttn& a = l.la;
            // heads in memory: the unrotated part, then the rotated one, each padded
            auto heads = [&](int k, int per0, int pad0, int per1, int pad1) {
                s[k].place_rows = a.heads * (pad0 + pad1);
                for (int h = 0; h < a.heads; h++) {
                    for (int d = 0; d < per0; d++) s[k].place.push_back(h * (pad0 + pad1) + d);
                    for (int d = 0; d < per1; d++) s[k].place.push_back(h * (pad0 + pad1) + pad0 + d);
                }
            };
            mat(MG_SLOT_LA_DQ, l.proj, 0, a.q_rank, W); mat(MG_SLOT_LA_DKV, l.proj, a.q_rank, a.rank + a.rot, W);
            vec(MG_SLOT_LA_DQNORM, l.dq_norm, a.q_rank); vec(MG_SLOT_LA_DKVNORM, l.dkv_norm, a.rank);
            mat(MG_SLOT_LA_UQ, l.uq, 0, a.heads * (a.dim + a.rot), a.q_rank); heads(MG_SLOT_LA_UQ, a.dim, a.dim_s, a.rot, a.rot_s);
            mat(MG_SLOT_LA_UK, l.uk, 0, a.heads * a.dim, a.rank); heads(MG_SLOT_LA_UK, a.dim, a.dim_s, 0, 0);
            mat(MG_SLOT_LA_UV, l.uv, 0, a.heads * a.vdim, a.rank);
            mat(MG_SLOT_LA_O, l.o, 0, W, l.kout());
            a.q_norm = l.dq_norm; a.c_norm = l.dkv_norm; a.cos_tab = l.cos_tab; a.sin_tab = l.sin_tab;
            a.uk = (const __nv_bfloat16*)l.uk; a.uv = (const __nv_bfloat16*)l.uv;
        } else {
            const int n = l.kout();
            for (int k = 0; k < 5; k++) vec(MG_SLOT_WKV_MU + k, l.mu[k], W);
            for (int k = 0; k < 4; k++) mat(MG_SLOT_WKV_R + k, l.proj, k * n, n, W);
            mat(MG_SLOT_WKV_W1, l.proj, 4 * n, l.wk.rank, W); mat(MG_SLOT_WKV_W2, l.w2, 0, n, l.wk.rank);
            vec(MG_SLOT_WKV_W0, l.w0, n); vec(MG_SLOT_WKV_U, l.u, n); vec(MG_SLOT_WKV_NORM, l.wkv_norm, n);
            mat(MG_SLOT_WKV_O, l.o, 0, W, n);
            l.wk.w2 = (const __nv_bfloat16*)l.w2; l.wk.w0 = l.w0; l.wk.u = l.u; l.wk.norm = l.wkv_norm;
        }
        if (l.moe.experts) {
            Moe& e = l.moe;
            vec(MG_SLOT_NORM2, l.norm2, W); vec(MG_SLOT_LS2, l.ls2, W); vec(MG_SLOT_MOE_BIAS, l.moe_bias, e.experts);
            mat(MG_SLOT_MOE_ROUTER, l.router, 0, e.experts, W);
            mat(MG_SLOT_MOE_GATE, l.e_gate, 0, e.experts * e.ff, W); mat(MG_SLOT_MOE_UP, l.e_up, 0, e.experts * e.ff, W);
            mat(MG_SLOT_MOE_DOWN, l.e_down, 0, e.experts * W, e.ff);
            if (e.shared_ff) {
                mat(MG_SLOT_SHARED_SG, l.router, e.sg_col(), 1, W);
                mat(MG_SLOT_SHARED_GATE, l.router, e.sg_col() + 1, e.shared_ff, W);
                mat(MG_SLOT_SHARED_UP, l.router, e.sg_col() + 1 + e.shared_ff, e.shared_ff, W);
                mat(MG_SLOT_SHARED_DOWN, l.shared_down, 0, W, e.shared_ff);
            }
            e.bias = l.moe_bias; e.gate = l.e_gate; e.up = l.e_up; e.down = l.e_down; e.shared_down = l.shared_down;
        }
    }
    LayerSlot* s = &m.slots[(size_t)c.n_layers * MG_LAYER_SLOTS];
    s[0].rows = s[2].rows = c.vocab; s[0].cols = s[2].cols = W; s[0].mat = m.embed; s[2].mat = m.head;
    s[1].rows = 1; s[1].cols = W; s[1].vec = m.final_norm;
    if (c.loop_times) { s[3].rows = W; s[3].cols = 2 * W; s[3].mat = m.loop_in; }
}

// Tables that positions index: angles and position vectors in float64 on the host, narrowed to fp32.
int layered_tables(mg_engine* e) {
    Layered& m = *e->lm;
    const int W = m.c.width, n = m.c.max_seq;
    auto upload = [&](float* to, const std::vector<float>& v) { return cudaMemcpy(to, v.data(), v.size() * 4, cudaMemcpyHostToDevice); };
    std::vector<float*> done;
    for (LayerWeights& l : m.layers) {
        if (l.parallel()) {
            std::vector<float> sl(l.at.heads);
            for (int h = 0; h < l.at.heads; h++) sl[h] = (float)pow(2.0, -8.0 * (h + 1) / l.at.heads);
            MG_CUDA(e, upload(l.slopes, sl));
        } else if (l.c.mixer == MG_MIXER_LATENT && std::find(done.begin(), done.end(), l.cos_tab) == done.end()) {
            done.push_back(l.cos_tab);
            const int half = l.la.rot / 2;
            std::vector<float> cs((size_t)n * half), sn((size_t)n * half);
            for (int i = 0; i < half; i++) {
                const double f = pow(l.c.latent.rot_base, -2.0 * i / l.la.rot);
                for (int p = 0; p < n; p++) { cs[(size_t)p * half + i] = (float)cos(p * f); sn[(size_t)p * half + i] = (float)sin(p * f); }
            }
            MG_CUDA(e, upload(l.cos_tab, cs));
            MG_CUDA(e, upload(l.sin_tab, sn));
        }
    }
    if (m.c.positions == MG_POS_SINUSOID) {
        std::vector<double> f((W + 1) / 2);
        for (size_t i = 0; i < f.size(); i++) f[i] = pow(10000.0, -2.0 * (double)i / W);
        std::vector<float> tab((size_t)n * W);
        for (int p = 0; p < n; p++)
            for (int i = 0; i < W; i++) tab[(size_t)p * W + i] = (float)(i & 1 ? cos(p * f[i / 2]) : sin(p * f[i / 2]));
        MG_CUDA(e, upload(m.pos_tab, tab));
    }
    return MG_OK;
}

int layered_set(mg_engine* e, int idx, const void* data, size_t count, bool bf16) {
    Layered& m = *e->lm;
    if (!data || idx < 0 || idx >= (int)m.slots.size() || !m.slots[idx].rows) return fail(e, MG_ERR_ARG, "weight slot %d does not exist in this model", idx);
    LayerSlot& s = m.slots[idx];
    if (count != (size_t)s.rows * s.cols) return fail(e, MG_ERR_ARG, "weight slot %d wants %d x %d values, got %zu", idx, s.rows, s.cols, count);
    const float* f = static_cast<const float*>(data);
    const uint16_t* h = static_cast<const uint16_t*>(data);
    if (s.vec) {
        std::vector<float> v(count);
        for (size_t i = 0; i < count; i++) {
            if (bf16) { const uint32_t w = (uint32_t)h[i] << 16; memcpy(&v[i], &w, 4); }
            else v[i] = f[i];
        }
        if (!bf16 && s.rounds)              // multiplied on the tensor cores: kept as bf16, like every matrix
            for (float& x : v) x = __bfloat162float(__float2bfloat16_rn(x));
        MG_CUDA(e, cudaMemcpy(s.vec, v.data(), count * 4, cudaMemcpyHostToDevice));
    } else if (const size_t ld = pad_to(s.cols, 64); bf16 && ld == (size_t)s.cols && s.place.empty()) {
        MG_CUDA(e, cudaMemcpy(s.mat, h, count * 2, cudaMemcpyHostToDevice));
    } else {
        std::vector<uint16_t> v((size_t)(s.place.empty() ? s.rows : s.place_rows) * ld, 0);
        for (int r = 0; r < s.rows; r++) {
            uint16_t* to = v.data() + (s.place.empty() ? r : s.place[r]) * ld;
            for (int k = 0; k < s.cols; k++) {
                const size_t i = (size_t)r * s.cols + k;
                if (bf16) to[k] = h[i];
                else { const __nv_bfloat16 b = __float2bfloat16_rn(f[i]); memcpy(to + k, &b, 2); }
            }
        }
        MG_CUDA(e, cudaMemcpy(s.mat, v.data(), v.size() * 2, cudaMemcpyHostToDevice));
    }
    s.set = true;
    e->built = false;
    return MG_OK;
}

int layered_dequant(mg_engine* e, int idx, int row0, int nrows, float* out) {
    Layered& m = *e->lm;
    if (!out || idx < 0 || idx >= (int)m.slots.size() || !m.slots[idx].mat || !m.slots[idx].set || row0 < 0 || nrows < 0 ||
        row0 + nrows > m.slots[idx].rows)
        return fail(e, MG_ERR_ARG, "mg_dequant_rows: bad slot %d or rows", idx);
    const LayerSlot& s = m.slots[idx];
    const size_t ld = pad_to(s.cols, 64);
    std::vector<uint16_t> v((size_t)nrows * ld);
    if (s.place.empty()) {
        MG_CUDA(e, cudaMemcpy(v.data(), s.mat + (size_t)row0 * ld * 2, v.size() * 2, cudaMemcpyDeviceToHost));
    } else {
        for (int r = 0; r < nrows; r++)
            MG_CUDA(e, cudaMemcpy(v.data() + r * ld, s.mat + (size_t)s.place[row0 + r] * ld * 2, ld * 2, cudaMemcpyDeviceToHost));
    }
    for (int r = 0; r < nrows; r++)
        for (int k = 0; k < s.cols; k++) {
            const uint32_t w = (uint32_t)v[r * ld + k] << 16;
            memcpy(&out[(size_t)r * s.cols + k], &w, 4);
        }
    return MG_OK;
}

int layered_build(mg_engine* e) {
    for (size_t i = 0; i < e->lm->slots.size(); i++)
        if (e->lm->slots[i].rows && !e->lm->slots[i].set) return fail(e, MG_ERR_STATE, "mg_build: weight slot %zu has not been set", i);
    drop_graphs(e);
    e->built = true;
    return MG_OK;
}

// Recurrent state only moves forward: a step continues where the layers' state stands, or starts over at
// position 0 (the kernels read no earlier state there).
int layered_advance(mg_engine* e, int ls, int le, int pos, int n) {
    Layered& m = *e->lm;
    if (pos < 0 || n < 1 || pos + n > m.c.max_seq)
        return fail(e, MG_ERR_ARG, "positions %d..%d do not fit max_seq %d", pos, pos + n - 1, m.c.max_seq);
    for (int l = ls; l < le; l++)
        if (pos != 0 && pos != m.runs[l].next_pos)
            return fail(e, MG_ERR_STATE, "layer %d has seen %d tokens; a step at position %d cannot continue it", l, m.runs[l].next_pos, pos);
    for (int l = ls; l < le; l++) m.runs[l].next_pos = pos + n;
    return MG_OK;
}

void layered_reset(mg_engine* e) {
    for (LayerRun& r : e->lm->runs) r.next_pos = 0;
}

void layered_phase_shape(const mg_engine* e, int nitems, int* grid) { *grid = std::max(1, std::min((nitems + 7) / 8, 2 * e->num_sms)); }

// One token through the layer runs [ls, le) (+ head).  The residual sum after a sublayer is formed by the kernel
// that next reads it; its CTA 0 stores it into the other of the two hidden buffers, so that the others can
// still read the old one.  Where layers loop, the embedding is kept in x0 and every pass's input is a store too.
int enqueue_layered_step(mg_engine* e, cudaStream_t s, int ls, int le, int mode, int head) {
    Layered& m = *e->lm;
    const int W = m.c.width, L = (int)m.runs.size();
    const bool loop = m.c.loop_times > 0;
    if (le > L) le = L;
    const bool with_head = le >= L && head != HEAD_NONE;
    e->capture_kernels = 0;
    bool embed = mode == MODE_EMBED && ls == 0;
    int left = embed && !loop ? 1 : 0;          // stores of the residual on the way; the last one lands in e->h
    {
        bool sum = false;                       // a sum that nobody has formed yet
        for (int i = ls; i < le; i++) {
            const LayerWeights& l = m.layers[m.runs[i].layer];
            if (m.runs[i].begins) left += sum ? 0 : 1;
            left += l.parallel() ? (l.c.ffn_dim ? 2 : 1) : (l.moe.experts ? 2 : 1);
            sum = true;
        }
    }
    auto target = [&]() { left--; return left & 1 ? e->h2 : e->h; };
    float* cur = e->h;
    bool move = false;                          // the first reader copies what it reads out of the first target's way
    if (!embed && loop) {
        cudaMemcpyKind d2d = cudaMemcpyDeviceToDevice;
        if (ls == 0) {
            MG_CUDA(e, cudaMemcpyAsync(m.x0, e->h, (size_t)W * 4, d2d, s));
            cur = m.x0;
        } else if (left & 1) {
            MG_CUDA(e, cudaMemcpyAsync(e->h2, e->h, (size_t)W * 4, d2d, s));
            cur = e->h2;
        }
    } else if (!embed) {
        move = left & 1;
    }
    // what the next reader of the residual has to add
    int pending = PRO_X;
    const float *z0 = nullptr, *z1 = nullptr, *w0 = nullptr, *w1 = nullptr, *pw = nullptr;
    auto source = [&](PhaseArgs& a) {
        a.k_valid = W; a.K = m.kw; a.eps = m.c.norm_eps; a.st = e->st;
        if (embed) {
            a.pro = PRO_EMBED_POS; a.embed = WeightView{m.embed, nullptr}; a.embed_fmt = FMT_BF16; a.embed_ld = m.kw; a.pos_tab = m.pos_tab;
        } else {
            a.pro = pending; a.x_src = cur;
            if (pending != PRO_X) { a.z[0] = z0; a.z[1] = z1; a.z_w[0] = w0; a.z_w[1] = w1; a.post_w = pw; a.z_mult = m.c.residual_mult; }
        }
    };
    auto read_x = [&](PhaseArgs& a, const float* norm_w, int kind) {
        source(a);
        a.last_w = norm_w; a.last_kind = kind;
        if (embed) a.h_store = loop ? m.x0 : target();
        else if (pending != PRO_X) a.h_store = target();
        else if (move) a.h_store = e->h2;
        if (a.h_store) cur = a.h_store;
        embed = move = false;
        pending = PRO_X;
    };
    auto phase = [&](PhaseArgs& a, int epi) -> int {
        const int R = epi == EPI_LOGITS ? 4 : pick_rows_per_tile(e, a.rows[0]);
        a.nitems = (a.rows[0] + R - 1) / R;
        int grid;
        layered_phase_shape(e, a.nitems, &grid);
        MG_CUDA(e, launch(e, s, layered_phase(epi, R), grid, 256, ((size_t)a.K + 72) * sizeof(float), a));
        return MG_OK;
    };
    // a matrix on a plain vector, normed first where a weight is given
    auto product = [&](const float* x, int k, const uint8_t* w, int rows, float* out, const float* norm_w) -> int {
        PhaseArgs a{};
        a.pro = PRO_X; a.st = e->st; a.x_src = x; a.k_valid = k; a.K = pad_to(k, 64); a.eps = m.c.norm_eps;
        a.last_w = norm_w; a.last_kind = NORM_RMS;
        a.w[0] = WeightView{w, nullptr}; a.rows[0] = rows; a.out = out;
        return phase(a, EPI_STORE);
    };
    int rc;

    auto parallel_layer = [&](const LayerRun& run, LayerWeights& l) -> int {
        {   // every input projection of the mixer
            PhaseArgs a{};
            read_x(a, nullptr, 0);
            a.w[0] = WeightView{l.proj, nullptr}; a.rows[0] = l.cols.total; a.out = m.row;
            if ((rc = phase(a, EPI_STORE))) return rc;
        }
        MixerStep ms{};
        ms.at = run.at(l); ms.mem = run.mem(l); ms.c = l.cols; ms.proj = m.row; ms.st = e->st;
        ms.vslices = (l.mem.vdim + 31) / 32; ms.n_mem = l.mem.heads * ms.vslices; ms.splits = l.splits; ms.tile = l.tile;
        ms.part = m.part; ms.mem_o = m.mem_raw; ms.attn_out = m.attn; ms.mem_y = m.mem_y;
        MG_CUDA(e, launch_mixer_step(ms, m.f32, e->use_pdl, s));
        MG_CUDA(e, launch_mixer_join(ms, e->use_pdl, s));
        e->capture_kernels += 2;
        {   // both output projections
            PhaseArgs a{}, b{};
            const int R = pick_rows_per_tile(e, 2 * W);
            a.pro = b.pro = PRO_X; a.st = b.st = e->st;
            a.x_src = m.attn; a.k_valid = l.kat(); a.K = pad_to(l.kat(), 64); a.w[0] = WeightView{l.at_o, nullptr}; a.out = m.y[0];
            b.x_src = m.mem_y; b.k_valid = l.kmem(); b.K = pad_to(l.kmem(), 64); b.w[0] = WeightView{l.mem_o, nullptr}; b.out = m.y[1];
            a.rows[0] = b.rows[0] = W;
            a.nitems = b.nitems = (W + R - 1) / R;
            int ga;
            layered_phase_shape(e, a.nitems, &ga);
            const int gb = ga;
            MG_CUDA(e, launch(e, s, layered_phase_pair(R), ga + gb, 256, ((size_t)std::max(a.K, b.K) + 72) * sizeof(float), a, b, ga));
        }
        pending = PRO_POST_PAIR; z0 = m.y[0]; z1 = m.y[1]; w0 = l.at_out; w1 = l.mem_out; pw = l.norm1;
        if (l.c.ffn_dim) {
            PhaseArgs a{};
            read_x(a, nullptr, 0);
            a.w[0] = WeightView{l.up, nullptr}; a.rows[0] = l.c.ffn_dim; a.out = m.mid;
            if ((rc = phase(a, EPI_GELU))) return rc;
            if ((rc = product(m.mid, l.c.ffn_dim, l.down, W, m.z, nullptr))) return rc;
            pending = PRO_POST; z0 = m.z; z1 = nullptr; pw = l.norm2;
        }
        return MG_OK;
    };

    auto latent_mixer = [&](const LayerRun& run, LayerWeights& l) -> int {
        PhaseArgs a{};
        read_x(a, l.norm1, m.c.norm);
        a.w[0] = WeightView{l.proj, nullptr}; a.rows[0] = l.proj_rows(); a.out = m.row;
        if ((rc = phase(a, EPI_STORE))) return rc;
        if ((rc = product(m.row, l.la.q_rank, l.uq, l.la.heads * l.la.qrow(), m.q1, l.dq_norm))) return rc;
        LatentStep t{};
        t.at = run.la(l); t.st = e->st; t.tokens = 1; t.q = m.q1; t.down = m.row; t.qa = m.qa; t.splits = l.splits; t.tile = l.tile; t.group = l.group;
        t.part = m.lpart; t.ml = m.ml; t.out = m.attn; t.ld_out = l.kout();
        MG_CUDA(e, launch_latent_query(t, m.f32, e->use_pdl, s));
        MG_CUDA(e, launch_latent_attend(t, m.f32, e->use_pdl, s));
        MG_CUDA(e, launch_latent_value(t, true, e->use_pdl, s));
        e->capture_kernels += 3;
        return product(m.attn, l.kout(), l.o, W, m.z, nullptr);
    };

    auto wkv_mixer = [&](const LayerRun& run, LayerWeights& l) -> int {
        const int n = l.kout();
        PhaseArgs a{};
        read_x(a, l.norm1, m.c.norm);
        a.mix_prev = run.prev;
        PhaseParts p{};
        p.n = 5;
        const int R = pick_rows_per_tile(e, l.proj_rows());
        for (int k = 0; k < 5; k++) {
            p.rows[k] = k < 4 ? n : l.wk.rank;
            p.w[k] = WeightView{l.proj + (size_t)k * n * m.kw * 2, nullptr};
            p.out[k] = m.row + (size_t)k * n;
            p.mu[k] = l.mu[k];
            const int items = (p.rows[k] + R - 1) / R, most = std::max(1, (int)((long long)2 * e->num_sms * p.rows[k] / l.proj_rows()));
            p.first[k + 1] = p.first[k] + std::max(1, std::min((items + 7) / 8, most));
        }
        MG_CUDA(e, launch(e, s, layered_phase_parts(R), p.first[5], 256, ((size_t)a.K + 72) * sizeof(float), a, p));
        WkvStep t{};
        t.wk = run.wk(l); t.row = m.row; t.st = e->st; t.y = m.attn;
        MG_CUDA(e, launch_wkv_step(t, e->use_pdl, s));
        e->capture_kernels += 1;
        return product(m.attn, n, l.o, W, m.z, nullptr);
    };

    auto experts = [&](LayerWeights& l) -> int {
        PhaseArgs a{};
        read_x(a, l.norm2, m.c.norm);
        a.n_store = m.hn;
        a.w[0] = WeightView{l.router, nullptr}; a.rows[0] = l.router_rows(); a.out = m.rt;
        if ((rc = phase(a, EPI_STORE))) return rc;
        MoeStep t{};
        t.moe = l.moe; t.router = m.rt; t.h = m.hn; t.sel = m.esel; t.mid = m.emid; t.out = m.z;
        MG_CUDA(e, launch_moe_up(t, e->num_sms, e->use_pdl, s));
        MG_CUDA(e, launch_moe_down(t, e->num_sms, e->use_pdl, s));
        e->capture_kernels += 2;
        return MG_OK;
    };

    for (int i = ls; i < le; i++) {
        LayerRun& run = m.runs[i];
        LayerWeights& l = m.layers[run.layer];
        if (run.begins) {                       // x <- W_in [x; x0], x being the sum that is still to be formed
            PhaseArgs a{};
            source(a);
            if (embed) { a.h_store = m.x0; embed = false; }
            pending = PRO_X;
            a.cat = m.x0; a.K = m.kl;
            a.w[0] = WeightView{m.loop_in, nullptr}; a.rows[0] = W; a.out = target();
            if ((rc = phase(a, EPI_STORE))) return rc;
            cur = a.out;
        }
        if (l.parallel()) {
            if ((rc = parallel_layer(run, l))) return rc;
            continue;
        }
        if ((rc = l.c.mixer == MG_MIXER_LATENT ? latent_mixer(run, l) : wkv_mixer(run, l))) return rc;
        pending = PRO_ADD; z0 = m.z; w0 = l.ls1;
        if (!l.moe.experts) continue;
        if ((rc = experts(l))) return rc;
        pending = PRO_ADD; z0 = m.z; w0 = l.ls2;
    }
    if (with_head) {
        PhaseArgs a{};
        read_x(a, m.final_norm, m.c.norm);
        a.w[0] = WeightView{m.head, nullptr}; a.rows[0] = m.c.vocab;
        a.out = head == HEAD_LOGITS ? e->logits : nullptr;
        a.out_tokens = e->out_tokens;
        if ((rc = phase(a, EPI_LOGITS))) return rc;
    } else if (pending != PRO_X || embed) {
        ResolveArgs r{};
        read_x(r.p, nullptr, 0);
        r.p.h_store = nullptr;
        r.out = e->h;
        MG_CUDA(e, launch_resolve(r, e->use_pdl, s));
        e->capture_kernels += 1;
    }
    return MG_OK;
}

// out[n][ldc] = act W^T over bf16 weights; gelu writes activations instead.  ld: padded row length of both.
int layered_matmul(mg_engine* e, const void* act, int act_rows, int ld, const uint8_t* w, void* out, int ldc, int n, int rows, bool gelu) {
    Layered& m = *e->lm;
    e->launches += 1;
    if (m.f32) {
        GemmF32 g{};
        g.A = (const float*)act; g.lda = ld; g.W = w; g.ldw = ld; g.out = (float*)out; g.ldc = ldc; g.n = n; g.rows = rows; g.K = ld;
        g.epi = gelu ? F32_GELU : F32_STORE;
        MG_CUDA(e, launch_gemm_f32(g, e->stream));
        return MG_OK;
    }
    GemmTC g{};
    g.bn = rows > 64 ? 128 : 64;
    if (!make_tile_map(&g.a, act, ld, act_rows, 1, ld, (long long)act_rows * ld, 128) ||
        !make_tile_map(&g.b, w, ld, rows, 1, ld, (long long)rows * ld, g.bn))
        return fail(e, MG_ERR_CUDA, "tensor map of a %d x %d product failed", rows, ld);
    g.m = n; g.n = rows; g.k = ld; g.batch = 1; g.b_group = 1; g.causal_pos0 = -1;
    g.out = out; g.ldc = ldc; g.mode = gelu ? GEMM_GELU_BF16 : GEMM_F32; g.status = m.status;
    MG_CUDA(e, launch_gemm_tc(g, e->stream));
    return MG_OK;
}

// The same over `count` matrices of `rows` rows each, stacked: out columns [z * rows, (z + 1) * rows) = act z W_z^T,
// act z `stride` elements after the one before it.
int layered_matmul_batch(mg_engine* e, const void* act, long long stride, int act_rows, int ld, const uint8_t* w, float* out, int ldc, int n,
                         int rows, int count) {
    Layered& m = *e->lm;
    if (m.f32) {
        for (int z = 0; z < count; z++)
            if (int rc = layered_matmul(e, (const float*)act + z * stride, act_rows, ld, w + (size_t)z * rows * ld * 2, out + (size_t)z * rows, ldc, n, rows, false)) return rc;
        return MG_OK;
    }
    e->launches += 1;
    GemmTC g{};
    g.bn = rows > 64 ? 128 : 64;
    if (!make_tile_map(&g.a, act, ld, act_rows, count, ld, stride, 128) || !make_tile_map(&g.b, w, ld, rows, count, ld, (long long)rows * ld, g.bn))
        return fail(e, MG_ERR_CUDA, "tensor map of %d %d x %d products failed", count, rows, ld);
    g.m = n; g.n = rows; g.k = ld; g.batch = count; g.b_group = 1; g.causal_pos0 = -1;
    g.out = out; g.ldc = ldc; g.batch_c = rows; g.mode = GEMM_F32; g.status = m.status;
    MG_CUDA(e, launch_gemm_tc(g, e->stream));
    return MG_OK;
}

// The same for few columns, which too few CTAs would share: the columns of act are cut into slices whose products
// land in out[slice][n][ldc], for the reader to add in order.  Returns the number of slices in *slices.
int layered_matmul_thin(mg_engine* e, const void* act, int act_rows, int ld, const uint8_t* w, float* out, int ldc, int n, int rows, int* slices) {
    Layered& m = *e->lm;
    int S = m.f32 || rows > 64 ? 1 : kThinSlices;
    while (ld / 64 % S) S /= 2;
    *slices = S;
    if (S == 1) return layered_matmul(e, act, act_rows, ld, w, out, ldc, n, rows, false);
    e->launches += 1;
    const int k = ld / S;
    GemmTC g{};
    g.bn = 64;
    if (!make_tile_map(&g.a, act, k, act_rows, S, ld, k, 128) || !make_tile_map(&g.b, w, k, rows, S, ld, k, g.bn))
        return fail(e, MG_ERR_CUDA, "tensor map of a %d x %d product in %d slices failed", rows, ld, S);
    g.m = n; g.n = rows; g.k = k; g.batch = S; g.b_group = 1; g.causal_pos0 = -1;
    g.out = out; g.ldc = ldc; g.batch_c = (long long)n * ldc; g.mode = GEMM_F32; g.status = m.status;
    MG_CUDA(e, launch_gemm_tc(g, e->stream));
    return MG_OK;
}

// One gated feed-forward, or with `group` those of stacked experts, each tile of 128 rows its own: z = down(silu(gate
// act) * (up act)), fp32 or like activations.  ld, ffs: padded row lengths; `count` matrices are stacked.
int layered_glu(mg_engine* e, const void* act, int act_rows, int ld, const uint8_t* gate, const uint8_t* up, const uint8_t* down, int ff, int ffs,
                int count, const int* group, void* z, bool z_act, int n) {
    Layered& m = *e->lm;
    const int W = m.c.width;
    e->launches += m.f32 ? 3 : 2;
    if (m.f32) {
        GemmF32 g{};
        g.A = (const float*)act; g.lda = ld; g.W = gate; g.ldw = ld; g.out = m.glu; g.ldc = ffs; g.n = n; g.rows = ff; g.K = ld;
        g.group = group; g.group_stride = (long long)ff * ld;
        MG_CUDA(e, launch_gemm_f32(g, e->stream));
        g.W = up; g.out = (float*)m.xmid; g.epi = F32_SILU_MUL; g.aux = m.glu;
        MG_CUDA(e, launch_gemm_f32(g, e->stream));
        g = GemmF32{};
        g.A = (const float*)m.xmid; g.lda = ffs; g.W = down; g.ldw = ffs; g.out = (float*)z; g.ldc = W; g.n = n; g.rows = W; g.K = ffs;
        g.group = group; g.group_stride = (long long)W * ffs;
        MG_CUDA(e, launch_gemm_f32(g, e->stream));
        return MG_OK;
    }
    GemmTC g{};
    g.bn = 128; g.m = n; g.n = ff; g.k = ld; g.batch = 1; g.b_group = 1; g.causal_pos0 = -1; g.group = group;
    g.out = m.xmid; g.ldc = ffs; g.mode = GEMM_SILU_BF16; g.status = m.status;
    if (!make_tile_map(&g.a, act, ld, act_rows, 1, ld, (long long)act_rows * ld, 128) ||
        !make_tile_map(&g.b, gate, ld, ff, count, ld, (long long)ff * ld, 64) || !make_tile_map(&g.b2, up, ld, ff, count, ld, (long long)ff * ld, 64))
        return fail(e, MG_ERR_CUDA, "tensor map of a %d x %d feed-forward failed", ff, ld);
    MG_CUDA(e, launch_gemm_tc(g, e->stream));
    g.bn = W > 64 ? 128 : 64; g.n = W; g.k = ffs; g.out = z; g.ldc = W; g.mode = z_act ? GEMM_BF16 : GEMM_F32;
    if (!make_tile_map(&g.a, m.xmid, ffs, act_rows, 1, ffs, (long long)act_rows * ffs, 128) ||
        !make_tile_map(&g.b, down, ffs, W, count, ffs, (long long)W * ffs, g.bn))
        return fail(e, MG_ERR_CUDA, "tensor map of a %d x %d feed-forward failed", W, ffs);
    MG_CUDA(e, launch_gemm_tc(g, e->stream));
    return MG_OK;
}

// Rows of the two-branch mixer: normed input rows in m.act, the branches' outputs into m.yr.
int parallel_rows(mg_engine* e, const LayerRun& run, LayerWeights& l, int pos, int n) {
    Layered& m = *e->lm;
    const int W = m.c.width, kat = pad_to(l.kat(), 64), kmem = pad_to(l.kmem(), 64), np = pad_to(l.cols.total, 4);
    cudaStream_t s = e->stream;
    const GateAttn at = run.at(l);
    int rc;
    if ((rc = layered_matmul(e, m.act, m.max_rows, m.kw, l.proj, m.P, np, n, l.cols.total, false))) return rc;
    MG_CUDA(e, launch_qk_rows(at, m.P, np, l.cols.q, l.cols.k, pos, n, m.qh, m.f32, s));
    if (l.block_rows) {
        int k = 0;
        MG_CUDA(e, launch_gate_attn_tc(at, m.qh, pos, n, m.max_rows, m.aw, l.block_rows, m.vt, m.ao, kat, m.status, &k, s));
        e->launches += k - 1;
    } else {
        MG_CUDA(e, launch_gate_attn_rows(at, m.qh, pos, n, m.ao, kat, m.f32, s));
    }
    MG_CUDA(e, launch_mem_rows(run.mem(l), l.cols, m.P, np, pos, n, m.mw, m.my, kmem, m.f32, s));
    e->launches += 7;
    if ((rc = layered_matmul(e, m.ao, m.max_rows, kat, l.at_o, m.yr[0], W, n, W, false))) return rc;
    return layered_matmul(e, m.my, m.max_rows, kmem, l.mem_o, m.yr[1], W, n, W, false);
}

// Rows of latent attention: normed input rows in m.act, output rows into m.zr.
int latent_rows(mg_engine* e, const LayerRun& run, LayerWeights& l, int pos, int n) {
    Layered& m = *e->lm;
    const LatentAttn at = run.la(l);
    const int np = pad_to(l.proj_rows(), 4), kq = pad_to(at.q_rank, 64), ko = pad_to(l.kout(), 64), qrows = at.heads * at.qrow();
    cudaStream_t s = e->stream;
    int rc;
    if ((rc = layered_matmul(e, m.act, m.max_rows, m.kw, l.proj, m.P, np, n, l.proj_rows(), false))) return rc;
    MG_CUDA(e, launch_latent_rows(at, m.P, np, pos, n, m.cq, kq, m.f32, s));
    if ((rc = layered_matmul(e, m.cq, m.max_rows, kq, l.uq, m.q32, qrows, n, qrows, false))) return rc;
    if (l.latent_tc) {
        int k = 0;
        MG_CUDA(e, launch_latent_q_rows(at, m.q32, pos, n, m.qh, s));
        MG_CUDA(e, launch_latent_attn_tc(at, m.qh, pos, n, m.keys, m.vt, pad_to(m.c.max_seq, 64), m.ao, ko, m.status, &k, s));
        e->launches += 2 + k;
    } else {
        LatentStep t{};
        t.at = at; t.pos0 = pos; t.tokens = n; t.q = m.q32; t.qa = m.qa; t.splits = 1; t.tile = l.tile; t.group = l.group;
        t.part = m.lpart; t.ml = m.ml; t.out = m.ao; t.ld_out = ko;
        MG_CUDA(e, launch_latent_query(t, m.f32, false, s));
        MG_CUDA(e, launch_latent_attend(t, m.f32, false, s));
        MG_CUDA(e, launch_latent_value(t, m.f32, false, s));
        e->launches += 4;
    }
    return layered_matmul(e, m.ao, m.max_rows, ko, l.o, m.zr, m.c.width, n, m.c.width, false);
}

// Rows of the linear recurrence: normed input rows in m.hr (32-bit), output rows into m.zr.
int wkv_rows(mg_engine* e, const LayerRun& run, LayerWeights& l, int pos, int n) {
    Layered& m = *e->lm;
    const Wkv wk = run.wk(l);
    const int W = m.c.width, kw = m.kw, d = l.kout(), np = pad_to(l.proj_rows(), 4), ko = pad_to(d, 64);
    const long long stride = (long long)m.max_rows * kw;
    cudaStream_t s = e->stream;
    int rc;
    MG_CUDA(e, launch_wkv_mix(m.hr, run.prev, l.mu, pos, n, W, m.mix, kw, stride, m.f32, s));
    MG_CUDA(e, cudaMemcpyAsync(run.prev + (size_t)((pos + n) & 1) * W, m.hr + (size_t)(n - 1) * W, (size_t)W * 4, cudaMemcpyDeviceToDevice, s));
    if ((rc = layered_matmul_batch(e, m.mix, stride, m.max_rows, kw, l.proj, m.P, np, n, d, 4))) return rc;
    int slices;
    const int ldi = pad_to(wk.rank, 4);
    if ((rc = layered_matmul_thin(e, m.mix + 4 * stride * (m.f32 ? 4 : 2), m.max_rows, kw, l.proj + (size_t)4 * d * kw * 2, m.inner32, ldi, n, wk.rank, &slices))) return rc;
    // decays: the inner vector stays 32-bit, on the tensor cores as a high and a low part
    if (m.f32) {
        GemmF32 g{};
        g.A = m.inner32; g.lda = ldi; g.W = l.w2; g.ldw = wk.ld2; g.out = m.decay; g.ldc = d; g.n = n; g.rows = d; g.K = wk.rank;
        g.epi = F32_DECAY; g.bias = l.w0;
        MG_CUDA(e, launch_gemm_f32(g, s));
    } else {
        const int ld = 2 * wk.ld2;
        MG_CUDA(e, launch_wkv_inner(m.inner32, ldi, slices, wk.rank, n, m.inner, ld, s));
        GemmTC g{};
        g.bn = d > 64 ? 128 : 64;
        if (!make_tile_map(&g.a, m.inner, ld, m.max_rows, 1, ld, (long long)m.max_rows * ld, 128) ||
            !make_tile_map(&g.b, l.w2, wk.ld2, d, 1, wk.ld2, (long long)d * wk.ld2, g.bn))
            return fail(e, MG_ERR_CUDA, "tensor map of a %d x %d product failed", d, ld);
        g.m = n; g.n = d; g.k = ld; g.batch = 1; g.b_group = 1; g.causal_pos0 = -1; g.b_steps = wk.ld2 / 64;
        g.out = m.decay; g.ldc = d; g.mode = GEMM_DECAY_F32; g.bias = l.w0; g.status = m.status;
        MG_CUDA(e, launch_gemm_tc(g, s));
        e->launches += 1;
    }
    MG_CUDA(e, launch_wkv_rows(wk, m.P, np, m.decay, pos, n, m.wo, s));
    MG_CUDA(e, launch_head_norm_rows(wk.heads, wk.dim, wk.eps, wk.norm, m.P + (size_t)3 * d, np, GATE_SILU, n, m.wo, m.ao, ko, m.f32, s));
    e->launches += 4;
    return layered_matmul(e, m.ao, m.max_rows, ko, l.o, m.zr, W, n, W, false);
}

// Rows of the mixture of experts: normed input rows in m.act, output rows into m.zr.
int moe_rows(mg_engine* e, LayerWeights& l, int n) {
    Layered& m = *e->lm;
    const Moe& x = l.moe;
    const int cols = x.experts + (x.shared_ff ? 1 : 0), ldr = pad_to(cols, 4);
    MoeRows w = m.moe;
    w.tiles = moe_tiles(x, n);
    cudaStream_t s = e->stream;
    int rc;
    int slices;
    if ((rc = layered_matmul_thin(e, m.act, m.max_rows, m.kw, l.router, m.rtr, ldr, n, cols, &slices))) return rc;
    MG_CUDA(e, launch_moe_route(x, m.rtr, ldr, slices, n, m.act, m.f32, w, s));
    if ((rc = layered_glu(e, w.x, w.tiles * 128, m.kw, l.e_gate, l.e_up, l.e_down, x.ff, x.ffs, x.experts, w.group, w.y, true, w.tiles * 128))) return rc;
    if (x.shared_ff && (rc = layered_glu(e, m.act, m.max_rows, m.kw, l.router_row(x.sg_col() + 1), l.router_row(x.sg_col() + 1 + x.shared_ff),
                                         l.shared_down, x.shared_ff, x.shared_ffs, 1, nullptr, m.zr, false, n))) return rc;
    MG_CUDA(e, launch_moe_combine(x, n, w, m.zr, m.f32, s));
    e->launches += 4;
    return MG_OK;
}

// Tokens m.tokens[0..n) at positions pos.. through every layer; leaves the residual rows in m.x.
int layered_rows(mg_engine* e, int pos, int n) {
    Layered& m = *e->lm;
    const int W = m.c.width, kw = m.kw;
    cudaStream_t s = e->stream;
    int rc;
    MG_CUDA(e, launch_embed_rows(WeightView{m.embed, nullptr}, kw, m.pos_tab, m.tokens, pos, n, W, m.x, m.act, kw, m.f32, s));
    e->launches += 1;
    if (m.c.loop_times) MG_CUDA(e, cudaMemcpyAsync(m.x0r, m.x, (size_t)n * W * 4, cudaMemcpyDeviceToDevice, s));
    const float* scale = nullptr;               // m.zr, scaled by this vector, is still to be added
    auto resolve = [&](PrenormRows& a) -> int {
        a.x = m.x; a.n = n; a.width = W; a.eps = m.c.norm_eps; a.kind = m.c.norm;
        if (scale) { a.z = m.zr; a.ls = scale; a.mult = m.c.residual_mult; }
        scale = nullptr;
        e->launches += 1;
        MG_CUDA(e, launch_prenorm_rows(a, m.f32, s));
        return MG_OK;
    };
    auto normed = [&](const float* w, float* h) -> int {
        PrenormRows a{};
        a.norm_w = w; a.h = h; a.act = m.act; a.ld_act = kw;
        return resolve(a);
    };
    bool raw = true;                            // m.act holds the rows of m.x
    for (LayerRun& run : m.runs) {
        LayerWeights& l = m.layers[run.layer];
        if (run.begins) {
            PrenormRows a{};
            a.act = m.cat; a.ld_act = m.kl; a.cat = m.x0r;
            if ((rc = resolve(a))) return rc;
            if ((rc = layered_matmul(e, m.cat, m.max_rows, m.kl, m.loop_in, m.x, W, n, W, false))) return rc;
            raw = false;
        }
        if (l.parallel()) {
            if (!raw && (rc = normed(nullptr, nullptr))) return rc;
            if ((rc = parallel_rows(e, run, l, pos, n))) return rc;
            MG_CUDA(e, launch_post_rows(m.x, m.yr[0], m.yr[1], l.at_out, l.mem_out, l.norm1, m.c.norm_eps, n, W, m.act, kw, m.f32, s));
            e->launches += 1;
            raw = true;
            if (!l.c.ffn_dim) continue;
            const int kff = pad_to(l.c.ffn_dim, 64);
            if ((rc = layered_matmul(e, m.act, m.max_rows, kw, l.up, m.midr, kff, n, l.c.ffn_dim, true))) return rc;
            if ((rc = layered_matmul(e, m.midr, m.max_rows, kff, l.down, m.zr, W, n, W, false))) return rc;
            MG_CUDA(e, launch_post_rows(m.x, m.zr, nullptr, nullptr, nullptr, l.norm2, m.c.norm_eps, n, W, m.act, kw, m.f32, s));
            e->launches += 1;
            continue;
        }
        raw = false;
        const bool latent = l.c.mixer == MG_MIXER_LATENT;
        if ((rc = normed(l.norm1, latent ? nullptr : m.hr))) return rc;
        if ((rc = latent ? latent_rows(e, run, l, pos, n) : wkv_rows(e, run, l, pos, n))) return rc;
        scale = l.ls1;
        if (!l.moe.experts) continue;
        if ((rc = normed(l.norm2, nullptr))) return rc;
        if ((rc = moe_rows(e, l, n))) return rc;
        scale = l.ls2;
    }
    if (scale) {
        PrenormRows a{};
        if ((rc = resolve(a))) return rc;
    }
    return MG_OK;
}

// A portion of a prompt, in blocks of at most max_rows tokens.
int layered_forward(mg_engine* e, const int* tokens, int n, int pos, const int* want, int n_want, float* logits_out) {
    Layered& m = *e->lm;
    int rc;
    if ((rc = layered_advance(e, 0, (int)m.runs.size(), pos, n))) return rc;
    int w = 0;
    for (int b = 0; b < n; b += m.max_rows) {
        const int nb = std::min(m.max_rows, n - b);
        MG_CUDA(e, cudaStreamSynchronize(e->stream));                 // the pinned words are reused
        memcpy(e->pin_i + 8, tokens + b, (size_t)nb * 4);
        MG_CUDA(e, cudaMemcpyAsync(m.tokens, e->pin_i + 8, (size_t)nb * 4, cudaMemcpyHostToDevice, e->stream));
        if ((rc = layered_rows(e, pos + b, nb))) return rc;
        while (w < n_want && want[w] < b + nb) {
            int k = 0;
            MG_CUDA(e, cudaStreamSynchronize(e->stream));
            while (w + k < n_want && want[w + k] < b + nb && k < m.logit_rows) { e->pin_i[8 + k] = want[w + k] - b; k++; }
            MG_CUDA(e, cudaMemcpyAsync(m.want, e->pin_i + 8, (size_t)k * 4, cudaMemcpyHostToDevice, e->stream));
            MG_CUDA(e, launch_last_norm_rows(m.x, m.want, m.final_norm, m.c.norm, m.c.norm_eps, k, m.c.width, m.fin, m.kw, m.f32, e->stream));
            e->launches += 1;
            if ((rc = layered_matmul(e, m.fin, m.logit_rows, m.kw, m.head, m.logits, m.c.vocab, k, m.c.vocab, false))) return rc;
            MG_CUDA(e, cudaMemcpyAsync(logits_out + (size_t)w * m.c.vocab, m.logits, (size_t)k * m.c.vocab * 4, cudaMemcpyDeviceToHost, e->stream));
            w += k;
        }
    }
    return MG_OK;
}

}  // namespace
