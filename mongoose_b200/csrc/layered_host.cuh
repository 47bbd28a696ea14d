// Host side of layer-described models: buffers, weights, one token (a captured sequence of phase kernels,
// like enqueue_step's) and portions of a prompt.  Included by engine.cu, whose engine, arena, cursor,
// graph cache and stepping calls it shares.
#pragma once

struct LayerWeights {
    mg_layer_config c{};
    ProjCols cols{};
    int splits = 1, tile = 16;
    int block_rows = 0;                 // queries per block of the tensor-core attention; 0: CUDA-core kernel
    uint8_t *proj = nullptr, *at_o = nullptr, *mem_o = nullptr, *up = nullptr, *down = nullptr;
    float *norm1 = nullptr, *norm2 = nullptr, *at_out = nullptr, *mem_out = nullptr;
    float *q_norm = nullptr, *k_norm = nullptr, *talk = nullptr, *bias = nullptr, *slopes = nullptr;
    float *mem_norm = nullptr, *i_bias = nullptr, *f_bias = nullptr;
    GateAttn at{};
    MatMem mem{};
    int next_pos = 0;                   // tokens this layer's cache and state have seen
    int kat() const { return c.attn.heads * c.attn.dim; }
    int kmem() const { return c.mem.heads * c.mem.vdim; }
};

struct LayerSlot {
    int rows = 0, cols = 0;             // 0: the slot does not exist
    uint8_t* mat = nullptr;             // bf16 rows padded to pad_to(cols, 64)
    float* vec = nullptr;
    bool rounds = false;                // a small matrix among the vectors: held as fp32, rounded to bf16
    bool set = false;
};

struct Layered {
    mg_model_config c{};
    bool f32 = false;
    int kw = 0;                         // padded width
    std::vector<LayerWeights> layers;
    std::vector<LayerSlot> slots;
    uint8_t *embed = nullptr, *head = nullptr;
    float *final_norm = nullptr, *pos_tab = nullptr;
    // one token
    float *row = nullptr, *part = nullptr, *attn = nullptr, *mem_raw = nullptr, *mem_y = nullptr, *y[2] = {}, *z = nullptr, *mid = nullptr;
    // portions
    int max_rows = 0, logit_rows = 0;
    int *tokens = nullptr, *want = nullptr;
    float *x = nullptr, *P = nullptr, *yr[2] = {}, *zr = nullptr, *logits = nullptr;
    uint8_t *act = nullptr, *qh = nullptr, *ao = nullptr, *my = nullptr, *midr = nullptr, *fin = nullptr;
    uint8_t *aw = nullptr, *vt = nullptr;   // tensor-core attention: mixed weights of a query block, transposed keys
    MemRows mw{};
    int np = 0;                         // widest projection row
    int* status = nullptr;              // set by a wait inside a tensor-core kernel that ran out
};

namespace {

// Runs `take(pointer, bytes)` over every device buffer of the model, so that sizing the arena and
// carving it are one list.
template <typename F>
int layered_buffers(Layered& m, F take) {
    const mg_model_config& c = m.c;
    const int W = c.width, kw = m.kw, T = m.max_rows;
    const size_t as = m.f32 ? 4 : 2;
    int rc = 0;
    auto get = [&](auto** p, size_t count, size_t elem) {
        if (!rc) rc = take((void**)p, count * elem);
    };
    int hd = 1, kat = 1, kmem = 1, ff = 1, mh = 1;
    size_t u = 1, nu = 1, part = 1, aw = 1, vt = 1;
    for (LayerWeights& l : m.layers) {
        const mg_gate_attn_config& a = l.c.attn;
        const mg_mat_mem_config& r = l.c.mem;
        get(&l.proj, (size_t)l.cols.total * kw, 2);
        get(&l.at_o, (size_t)W * pad_to(l.kat(), 64), 2);
        get(&l.mem_o, (size_t)W * pad_to(l.kmem(), 64), 2);
        get(&l.norm1, W, 4); get(&l.at_out, W, 4); get(&l.mem_out, W, 4);
        if (l.c.ffn_dim) {
            get(&l.norm2, W, 4);
            get(&l.up, (size_t)l.c.ffn_dim * kw, 2);
            get(&l.down, (size_t)W * pad_to(l.c.ffn_dim, 64), 2);
        }
        get(&l.q_norm, a.dim, 4); get(&l.k_norm, a.dim, 4); get(&l.talk, (size_t)a.heads * a.heads, 4);
        get(&l.bias, a.heads, 4); get(&l.slopes, a.heads, 4);
        get(&l.mem_norm, l.kmem(), 4); get(&l.i_bias, r.heads, 4); get(&l.f_bias, r.heads, 4);
        get(&l.at.cache, (size_t)c.max_seq * a.kv_heads * l.at.dim_s, as);
        get(&l.at.cache_r, (size_t)c.max_seq * a.kv_heads, 4);
        get(&l.mem.S, (size_t)r.heads * r.dim * r.vdim, 4);
        get(&l.mem.nrm, (size_t)2 * r.heads * r.dim, 4);
        get(&l.mem.m, (size_t)2 * r.heads, 4);
        hd = std::max(hd, a.heads * l.at.dim_s);
        kat = std::max(kat, pad_to(l.kat(), 64)); kmem = std::max(kmem, pad_to(l.kmem(), 64));
        ff = std::max(ff, pad_to(l.c.ffn_dim, 64)); mh = std::max(mh, r.heads);
        const size_t chunks = (T + kMemChunk - 1) / kMemChunk;
        u = std::max(u, chunks * r.heads * r.dim * r.vdim); nu = std::max(nu, chunks * r.heads * r.dim);
        if (l.block_rows) {
            aw = std::max(aw, (size_t)a.heads * l.block_rows * pad_to(c.max_seq, 64));
            vt = std::max(vt, (size_t)a.kv_heads * a.dim * pad_to(c.max_seq, 64));
        }
        part = std::max(part, (size_t)l.splits * a.heads * l.at.dim_s);
    }
    get(&m.embed, (size_t)c.vocab * kw, 2); get(&m.head, (size_t)c.vocab * kw, 2);
    get(&m.final_norm, W, 4); get(&m.pos_tab, (size_t)c.max_seq * W, 4);
    get(&m.row, m.np, 4); get(&m.part, part, 4); get(&m.attn, kat, 4);
    get(&m.mem_raw, kmem, 4); get(&m.mem_y, kmem, 4); get(&m.y[0], W, 4); get(&m.y[1], W, 4); get(&m.z, W, 4); get(&m.mid, ff, 4);
    get(&m.status, 1, 4); get(&m.tokens, T, 4); get(&m.want, T, 4);
    get(&m.x, (size_t)T * W, 4); get(&m.P, (size_t)T * m.np, 4);
    get(&m.yr[0], (size_t)T * W, 4); get(&m.yr[1], (size_t)T * W, 4); get(&m.zr, (size_t)T * W, 4);
    get(&m.logits, (size_t)m.logit_rows * c.vocab, 4);
    get(&m.act, (size_t)T * kw, as); get(&m.qh, (size_t)T * hd, as); get(&m.ao, (size_t)T * kat, as);
    get(&m.my, (size_t)T * kmem, as); get(&m.midr, (size_t)T * ff, as); get(&m.fin, (size_t)m.logit_rows * kw, as);
    get(&m.aw, aw, 2); get(&m.vt, vt, 2);
    get(&m.mw.b, (size_t)mh * T, 8); get(&m.mw.ig, (size_t)mh * T, 4); get(&m.mw.mm, (size_t)mh * T, 4); get(&m.mw.m0, mh, 4);
    get(&m.mw.g, (size_t)mh * ((T + kMemChunk - 1) / kMemChunk), 4);
    get(&m.mw.U, u, 4); get(&m.mw.nU, nu, 4); get(&m.mw.o, (size_t)T * kmem, 4);
    return rc;
}

// Shapes, slots and kernel arguments; MG_ERR_ARG / MG_ERR_UNSUPPORTED with a reason in *why.
int layered_shapes(Layered& m, int sms, std::string* why) {
    const mg_model_config& c = m.c;
    if (c.width <= 0 || c.vocab <= 0 || c.n_layers <= 0 || c.max_seq <= 0 || !(c.norm_eps >= 0.f) ||
        (c.math != MG_MATH_BF16 && c.math != MG_MATH_F32)) { *why = "bad model sizes"; return MG_ERR_ARG; }
    m.f32 = c.math == MG_MATH_F32;
    m.kw = pad_to(c.width, 64);
    int kmax = m.kw;
    m.max_rows = std::min(c.max_seq, 2048);
    m.logit_rows = std::max(1, std::min(std::min(128, m.max_rows), (int)((64u << 20) / ((size_t)c.vocab * 4))));
    for (LayerWeights& l : m.layers) {
        const mg_gate_attn_config& a = l.c.attn;
        const mg_mat_mem_config& r = l.c.mem;
        if (l.c.mixer != MG_MIXER_PARALLEL || a.heads <= 0 || a.kv_heads <= 0 || a.heads % a.kv_heads || a.dim <= 0 || a.temp_every <= 0 ||
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
        m.np = std::max(m.np, pad_to(o, 4));
        kmax = std::max(std::max(kmax, pad_to(l.kat(), 64)), std::max(pad_to(l.kmem(), 64), pad_to(l.c.ffn_dim, 64)));
    }
    // the phase kernels stage a whole input vector per CTA
    if (kmax > 48 * 1024) { *why = "a matrix with rows of more than 49152 values"; return MG_ERR_UNSUPPORTED; }
    if (layered_phase_smem(((size_t)kmax + 72) * sizeof(float)) != cudaSuccess) { *why = "kernel attributes"; return MG_ERR_CUDA; }
    return MG_OK;
}

void layered_slots(Layered& m) {
    const mg_model_config& c = m.c;
    const int W = c.width;
    m.slots.assign((size_t)c.n_layers * MG_LAYER_SLOTS + 3, LayerSlot{});
    for (int i = 0; i < c.n_layers; i++) {
        LayerWeights& l = m.layers[i];
        LayerSlot* s = &m.slots[(size_t)i * MG_LAYER_SLOTS];
        auto vec = [&](int k, float* p, int n) { s[k].rows = 1; s[k].cols = n; s[k].vec = p; };
        auto mat = [&](int k, uint8_t* p, int row0, int rows, int cols) {
            s[k].rows = rows; s[k].cols = cols; s[k].mat = p + (size_t)row0 * pad_to(cols, 64) * 2;
        };
        const mg_gate_attn_config& a = l.c.attn;
        const mg_mat_mem_config& r = l.c.mem;
        vec(MG_SLOT_NORM1, l.norm1, W);
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
    }
    LayerSlot* s = &m.slots[(size_t)c.n_layers * MG_LAYER_SLOTS];
    s[0].rows = s[2].rows = c.vocab; s[0].cols = s[2].cols = W; s[0].mat = m.embed; s[2].mat = m.head;
    s[1].rows = 1; s[1].cols = W; s[1].vec = m.final_norm;
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
    } else {
        const size_t ld = pad_to(s.cols, 64);
        std::vector<uint16_t> v((size_t)s.rows * ld, 0);
        for (int r = 0; r < s.rows; r++)
            for (int k = 0; k < s.cols; k++) {
                const size_t i = (size_t)r * s.cols + k;
                if (bf16) v[r * ld + k] = h[i];
                else { const __nv_bfloat16 b = __float2bfloat16_rn(f[i]); memcpy(&v[r * ld + k], &b, 2); }
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
    MG_CUDA(e, cudaMemcpy(v.data(), s.mat + (size_t)row0 * ld * 2, v.size() * 2, cudaMemcpyDeviceToHost));
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
        if (pos != 0 && pos != m.layers[l].next_pos)
            return fail(e, MG_ERR_STATE, "layer %d has seen %d tokens; a step at position %d cannot continue it", l, m.layers[l].next_pos, pos);
    for (int l = ls; l < le; l++) m.layers[l].next_pos = pos + n;
    return MG_OK;
}

void layered_reset(mg_engine* e) {
    for (LayerWeights& l : e->lm->layers) l.next_pos = 0;
}

void layered_phase_shape(const mg_engine* e, int nitems, int* grid) { *grid = std::max(1, std::min((nitems + 7) / 8, 2 * e->num_sms)); }

// One token through layers [ls, le) (+ head): five fused kernels and the mixer's join per layer.  The
// residual sum after a sublayer is formed by the kernel that next reads it; its CTA 0 stores it into the
// other of the two hidden buffers, so that the others can still read the old one.
int enqueue_layered_step(mg_engine* e, cudaStream_t s, int ls, int le, int mode, int head) {
    Layered& m = *e->lm;
    const int W = m.c.width, L = m.c.n_layers;
    if (le > L) le = L;
    const bool with_head = le >= L && head != HEAD_NONE;
    e->capture_kernels = 0;
    int sums = 0;                               // residual sums formed on the way
    for (int l = ls; l < le; l++) sums += m.layers[l].c.ffn_dim ? 2 : 1;
    float* bufs[2] = {e->h, e->h2};
    int at = (mode == MODE_EMBED && ls == 0) ? (sums & 1) : 0;   // the last sum lands in e->h
    bool embed = mode == MODE_EMBED && ls == 0, move = !embed && (sums & 1);
    // what the next reader of the residual has to add
    int pending = PRO_X;
    const float *z0 = nullptr, *z1 = nullptr, *w0 = nullptr, *w1 = nullptr, *pw = nullptr;
    auto read_x = [&](PhaseArgs& a) {
        a.k_valid = W; a.K = m.kw; a.eps = m.c.norm_eps; a.st = e->st;
        if (embed) {
            a.pro = PRO_EMBED_POS; a.embed = WeightView{m.embed, nullptr}; a.embed_fmt = FMT_BF16; a.pos_tab = m.pos_tab;
            a.h_store = bufs[at];
            embed = false;
        } else if (pending == PRO_X) {
            a.pro = PRO_X; a.x_src = bufs[at];
            if (move) { a.h_store = bufs[at ^ 1]; at ^= 1; move = false; }
        } else {
            a.pro = pending; a.x_src = bufs[at]; a.z[0] = z0; a.z[1] = z1; a.z_w[0] = w0; a.z_w[1] = w1; a.post_w = pw;
            a.h_store = bufs[at ^ 1];
            at ^= 1;
        }
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
    int rc;
    for (int i = ls; i < le; i++) {
        LayerWeights& l = m.layers[i];
        {   // every input projection of the mixer
            PhaseArgs a{};
            read_x(a);
            a.w[0] = WeightView{l.proj, nullptr}; a.rows[0] = l.cols.total; a.out = m.row;
            if ((rc = phase(a, EPI_STORE))) return rc;
        }
        MixerStep ms{};
        ms.at = l.at; ms.mem = l.mem; ms.c = l.cols; ms.proj = m.row; ms.st = e->st;
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
            read_x(a);
            a.w[0] = WeightView{l.up, nullptr}; a.rows[0] = l.c.ffn_dim; a.out = m.mid;
            if ((rc = phase(a, EPI_GELU))) return rc;
            PhaseArgs b{};
            b.pro = PRO_X; b.st = e->st; b.x_src = m.mid; b.k_valid = l.c.ffn_dim; b.K = pad_to(l.c.ffn_dim, 64);
            b.w[0] = WeightView{l.down, nullptr}; b.rows[0] = W; b.out = m.z;
            if ((rc = phase(b, EPI_STORE))) return rc;
            pending = PRO_POST; z0 = m.z; z1 = nullptr; pw = l.norm2;
        }
    }
    if (with_head) {
        PhaseArgs a{};
        read_x(a);
        a.last_w = m.final_norm;
        a.w[0] = WeightView{m.head, nullptr}; a.rows[0] = m.c.vocab;
        a.out = head == HEAD_LOGITS ? e->logits : nullptr;
        a.out_tokens = e->out_tokens;
        if ((rc = phase(a, EPI_LOGITS))) return rc;
    } else if (pending != PRO_X || embed) {
        ResolveArgs r{};
        read_x(r.p);
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
        MG_CUDA(e, launch_gemm_f32((const float*)act, ld, w, ld, (float*)out, ldc, n, rows, ld, gelu, e->stream));
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

// Tokens m.tokens[0..n) at positions pos.. through every layer; leaves the residual rows in m.x.
int layered_rows(mg_engine* e, int pos, int n) {
    Layered& m = *e->lm;
    const int W = m.c.width, kw = m.kw;
    cudaStream_t s = e->stream;
    int rc;
    MG_CUDA(e, launch_embed_rows(WeightView{m.embed, nullptr}, kw, m.pos_tab, m.tokens, pos, n, W, m.x, m.act, kw, m.f32, s));
    e->launches += 1;
    for (LayerWeights& l : m.layers) {
        const int kat = pad_to(l.kat(), 64), kmem = pad_to(l.kmem(), 64), kff = pad_to(l.c.ffn_dim, 64), np = pad_to(l.cols.total, 4);
        if ((rc = layered_matmul(e, m.act, m.max_rows, kw, l.proj, m.P, np, n, l.cols.total, false))) return rc;
        MG_CUDA(e, launch_qk_rows(l.at, m.P, np, l.cols.q, l.cols.k, pos, n, m.qh, m.f32, s));
        if (l.block_rows) {
            int k = 0;
            MG_CUDA(e, launch_gate_attn_tc(l.at, m.qh, pos, n, m.max_rows, m.aw, l.block_rows, m.vt, m.ao, kat, m.status, &k, s));
            e->launches += k - 1;
        } else {
            MG_CUDA(e, launch_gate_attn_rows(l.at, m.qh, pos, n, m.ao, kat, m.f32, s));
        }
        MG_CUDA(e, launch_mem_rows(l.mem, l.cols, m.P, np, pos, n, m.mw, m.my, kmem, m.f32, s));
        e->launches += 7;
        if ((rc = layered_matmul(e, m.ao, m.max_rows, kat, l.at_o, m.yr[0], W, n, W, false))) return rc;
        if ((rc = layered_matmul(e, m.my, m.max_rows, kmem, l.mem_o, m.yr[1], W, n, W, false))) return rc;
        MG_CUDA(e, launch_post_rows(m.x, m.yr[0], m.yr[1], l.at_out, l.mem_out, l.norm1, m.c.norm_eps, n, W, m.act, kw, m.f32, s));
        e->launches += 1;
        if (!l.c.ffn_dim) continue;
        if ((rc = layered_matmul(e, m.act, m.max_rows, kw, l.up, m.midr, kff, n, l.c.ffn_dim, true))) return rc;
        if ((rc = layered_matmul(e, m.midr, m.max_rows, kff, l.down, m.zr, W, n, W, false))) return rc;
        MG_CUDA(e, launch_post_rows(m.x, m.zr, nullptr, nullptr, nullptr, l.norm2, m.c.norm_eps, n, W, m.act, kw, m.f32, s));
        e->launches += 1;
    }
    return MG_OK;
}

// A portion of a prompt, in blocks of at most max_rows tokens.
int layered_forward(mg_engine* e, const int* tokens, int n, int pos, const int* want, int n_want, float* logits_out) {
    Layered& m = *e->lm;
    int rc;
    if ((rc = layered_advance(e, 0, m.c.n_layers, pos, n))) return rc;
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
            MG_CUDA(e, launch_last_norm_rows(m.x, m.want, m.final_norm, m.c.norm_eps, k, m.c.width, m.fin, m.kw, m.f32, e->stream));
            e->launches += 1;
            if ((rc = layered_matmul(e, m.fin, m.logit_rows, m.kw, m.head, m.logits, m.c.vocab, k, m.c.vocab, false))) return rc;
            MG_CUDA(e, cudaMemcpyAsync(logits_out + (size_t)w * m.c.vocab, m.logits, (size_t)k * m.c.vocab * 4, cudaMemcpyDeviceToHost, e->stream));
            w += k;
        }
    }
    return MG_OK;
}

}  // namespace
