// Layer-stack models: weights, buffers and the pass (see stack.cuh).
#include "stack.cuh"

#include <algorithm>
#include <cmath>

#include "gemm.cuh"
#include "matrix_memory.cuh"
#include "stack_attention.cuh"

namespace ctox {

constexpr uint32_t kDefaultPass = 2048, kHeadRowsLong = 64;

namespace {

uint32_t round_up(uint32_t v, uint32_t to) { return (v + to - 1) / to * to; }

ctox_status dense_alloc(ctox_exec *e, DenseMat *d, uint64_t rows, uint64_t cols) {
    if (d->w) return CTOX_OK;
    d->rows = (uint32_t)rows;
    d->cols = (uint32_t)cols;
    d->ld = round_up((uint32_t)cols, 8);
    return xalloc(e, (void **)&d->w, (size_t)rows * d->ld * 2, false);
}

// One tensor as the file holds it, and where it goes.
struct Placement {
    uint64_t rows = 0, cols = 0;
    struct To {
        DenseMat *mat;
        uint64_t mat_rows, mat_cols;  // of the whole destination
        uint32_t row0;
        PadAxis ra, ca;
        uint32_t transpose_group, transpose_cols;
        uint32_t fill_rows;  // rows a synthetic fill writes (0: all of the destination)
    } to[2];
    int n = 0;
    uint64_t *loaded = nullptr;
};
PadAxis plain_axis(uint64_t n) { return PadAxis{(uint32_t)n, (uint32_t)n, 0, (uint32_t)n}; }
PadAxis head_axis(uint32_t per_head, uint32_t padded) { return PadAxis{per_head, per_head, 0, padded}; }

uint64_t fan_rows_of(const StackLayer &L) {
    const ctox_layer_config &c = L.c;
    if (c.mixer == CTOX_MIXER_LATENT_ATTENTION) return (uint64_t)c.q_rank + (c.kv_from < 0 ? c.kv_rank + c.rot_dim : 0);
    if (c.mixer == CTOX_MIXER_GROUPED_ATTENTION) return (uint64_t)(c.heads + c.kv_heads) * c.dim + (uint64_t)c.kv_heads * c.vdim;
    return (uint64_t)L.gate_row + 2ull * c.heads;
}

bool place(ctox_exec *e, uint32_t layer, uint32_t tensor, Placement *p) {
    StackModel *s = e->stack;
    const uint32_t H = s->c.hidden_size;
    auto whole = [&](DenseMat *m, uint64_t rows, uint64_t cols) {
        p->rows = rows;
        p->cols = cols;
        p->to[0] = {m, rows, cols, 0, plain_axis(rows), plain_axis(cols), 0, 0, 0};
        p->n = 1;
        return true;
    };
    if (layer == CTOX_LAYER_GLOBAL) {
        p->loaded = &s->loaded;
        if (tensor == CTOX_T_EMBED) return whole(&s->embed, s->c.vocab_size, H);
        if (tensor == CTOX_T_LM_HEAD) return !s->c.tied_head && whole(&s->head, s->c.vocab_size, H);
        return false;
    }
    if (layer >= s->layers.size()) return false;
    StackLayer &L = s->layers[layer];
    const ctox_layer_config &c = L.c;
    p->loaded = &L.loaded;
    const bool latent = c.mixer == CTOX_MIXER_LATENT_ATTENTION, memory = c.mixer == CTOX_MIXER_MATRIX_MEMORY,
               glu = c.mlp == CTOX_MLP_CLAMPED_GLU;
    const uint64_t fan_rows = fan_rows_of(L);
    // `rows` rows of the projection from `row0` on, in heads of `per_head` padded to `padded`
    auto in_fan = [&](uint64_t heads, uint32_t per_head, uint32_t padded, uint64_t row0) {
        whole(&L.fan, heads * per_head, H);
        p->to[0].mat_rows = fan_rows;
        p->to[0].row0 = (uint32_t)row0;
        p->to[0].ra = head_axis(per_head, padded);
        p->to[0].fill_rows = (uint32_t)(heads * padded);
        return true;
    };
    // every second row of the gated feed-forward's matrix
    auto interleaved = [&](uint32_t first) {
        whole(&L.up, c.ff, H);
        p->to[0].mat_rows = 2ull * c.ff;
        p->to[0].row0 = first;
        p->to[0].ra = PadAxis{1, 1, 0, 2};
        p->to[0].fill_rows = 2 * c.ff - first;
        return true;
    };
    const uint64_t kv_heads = memory ? c.heads : c.kv_heads;
    const uint32_t dim_to = memory ? L.dim_pad : c.dim, vdim_to = memory ? L.vdim_pad : c.vdim;
    const uint64_t k_row = (uint64_t)c.heads * dim_to, v_row = k_row + kv_heads * dim_to;
    switch (tensor) {
        case CTOX_T_MIX_Q: return !latent && in_fan(c.heads, c.dim, dim_to, 0);
        case CTOX_T_MIX_K: return !latent && in_fan(kv_heads, c.dim, dim_to, k_row);
        case CTOX_T_MIX_V: return !latent && in_fan(kv_heads, c.vdim, vdim_to, v_row);
        case CTOX_T_MIX_GATE: return memory && in_fan(c.heads, c.vdim, vdim_to, v_row + (uint64_t)c.heads * vdim_to);
        case CTOX_T_MEM_IN: return memory && in_fan(c.heads, 1, 1, L.gate_row);
        case CTOX_T_MEM_FORGET: return memory && in_fan(c.heads, 1, 1, L.gate_row + c.heads);
        case CTOX_T_MLP_GATE: return glu && interleaved(0);
        case CTOX_T_MLP_UP:
            if (glu) return interleaved(1);
            return c.mlp != CTOX_MLP_NONE && whole(&L.up, c.ff, H);
        case CTOX_T_MLP_DOWN: return c.mlp != CTOX_MLP_NONE && whole(&L.down, H, c.ff);
        case CTOX_T_ATTN_O:
            whole(&L.o, H, (uint64_t)c.heads * c.vdim);
            p->to[0].mat_cols = (uint64_t)c.heads * L.vdim_pad;
            p->to[0].ca = head_axis(c.vdim, L.vdim_pad);
            return true;
        default:
            if (!latent) return false;
    }
    switch (tensor) {
        case CTOX_T_Q_DOWN:
            whole(&L.fan, c.q_rank, H);
            p->to[0].mat_rows = fan_rows;
            p->to[0].fill_rows = c.q_rank;
            return true;
        case CTOX_T_KV_DOWN:
            if (c.kv_from >= 0) return false;
            whole(&L.fan, c.kv_rank + c.rot_dim, H);
            p->to[0].mat_rows = fan_rows;
            p->to[0].row0 = c.q_rank;
            p->to[0].fill_rows = c.kv_rank + c.rot_dim;
            return true;
        case CTOX_T_Q_UP:
            whole(&L.q_up, (uint64_t)c.heads * (c.dim + c.rot_dim), c.q_rank);
            p->to[0].mat_rows = (uint64_t)c.heads * L.head_w;
            p->to[0].ra = PadAxis{c.dim + c.rot_dim, c.dim, L.dim_pad, L.head_w};
            return true;
        case CTOX_T_K_UP:
            whole(&L.k_up_t, (uint64_t)c.heads * c.dim, c.kv_rank);
            p->to[0].mat_rows = (uint64_t)c.heads * L.kv_pad;
            p->to[0].mat_cols = L.dim_pad;
            p->to[0].ra = head_axis(c.dim, L.dim_pad);
            p->to[0].transpose_group = L.dim_pad;
            p->to[0].transpose_cols = L.kv_pad;
            if (s->pass_cap > kDensePass) {
                p->to[1] = {&L.k_up, (uint64_t)c.heads * L.dim_pad, L.kv_pad, 0, head_axis(c.dim, L.dim_pad),
                            plain_axis(c.kv_rank), 0, 0, 0};
                p->n = 2;
            }
            return true;
        case CTOX_T_V_UP:
            whole(&L.v_up, (uint64_t)c.heads * c.vdim, c.kv_rank);
            p->to[0].mat_rows = (uint64_t)c.heads * L.vdim_pad;
            p->to[0].mat_cols = L.kv_pad;
            p->to[0].ra = head_axis(c.vdim, L.vdim_pad);
            return true;
        default: return false;
    }
}

uint64_t bit(uint32_t tensor) { return 1ull << tensor; }

uint64_t layer_needs(const StackModel *s, const StackLayer &L) {
    const ctox_layer_config &c = L.c;
    uint64_t m = bit(CTOX_T_INPUT_NORM) | bit(CTOX_T_ATTN_O);
    if (s->c.out_norms) m |= bit(CTOX_T_MIX_OUT_NORM);
    if (c.mixer == CTOX_MIXER_LATENT_ATTENTION) {
        m |= bit(CTOX_T_Q_DOWN) | bit(CTOX_T_Q_DOWN_NORM) | bit(CTOX_T_Q_UP) | bit(CTOX_T_K_UP) | bit(CTOX_T_V_UP);
        if (c.kv_from < 0) m |= bit(CTOX_T_KV_DOWN) | bit(CTOX_T_KV_DOWN_NORM);
    } else {
        m |= bit(CTOX_T_MIX_Q) | bit(CTOX_T_MIX_K) | bit(CTOX_T_MIX_V);
    }
    if (c.mixer == CTOX_MIXER_GROUPED_ATTENTION) {
        if (c.attn & CTOX_ATTN_BIAS)
            m |= bit(CTOX_T_MIX_Q_BIAS) | bit(CTOX_T_MIX_K_BIAS) | bit(CTOX_T_MIX_V_BIAS) | bit(CTOX_T_MIX_O_BIAS);
        if (c.attn & CTOX_ATTN_QK_NORM) m |= bit(CTOX_T_Q_NORM) | bit(CTOX_T_K_NORM);
        if (c.attn & CTOX_ATTN_SINK) m |= bit(CTOX_T_ATTN_SINK);
        if (L.mixes_values) m |= bit(CTOX_T_V_MIX);
    }
    if (c.mixer == CTOX_MIXER_MATRIX_MEMORY)
        m |= bit(CTOX_T_MIX_GATE) | bit(CTOX_T_MIX_HEAD_NORM) | bit(CTOX_T_MEM_IN) | bit(CTOX_T_MEM_IN_BIAS) |
             bit(CTOX_T_MEM_FORGET) | bit(CTOX_T_MEM_FORGET_BIAS);
    if (c.mlp != CTOX_MLP_NONE) {
        m |= bit(CTOX_T_POST_NORM) | bit(CTOX_T_MLP_UP) | bit(CTOX_T_MLP_DOWN);
        if (c.mlp == CTOX_MLP_CLAMPED_GLU) m |= bit(CTOX_T_MLP_GATE);
        if (s->c.out_norms) m |= bit(CTOX_T_MLP_OUT_NORM);
    }
    return m;
}
uint64_t global_needs(const StackModel *s) {
    return bit(CTOX_T_EMBED) | bit(CTOX_T_FINAL_NORM) | (s->c.tied_head ? 0 : bit(CTOX_T_LM_HEAD));
}
const DenseMat &head_of(const StackModel *s) { return s->c.tied_head ? s->embed : s->head; }

MatrixMemory memory_args(const StackModel *s, const StackLayer &L) {
    return MatrixMemory{L.c.heads, L.c.dim,       L.c.vdim,  L.dim_pad, L.vdim_pad, L.c.gate_cap, s->c.norm_eps,
                        L.in_bias, L.forget_bias, L.head_norm, L.state, L.top};
}

}  // namespace

ctox_status stack_create(ctox_ctx *ctx, const ctox_stack_config *c, const ctox_layer_config *layers, ctox_exec **out) {
    if (ctx->tp_world > 1)
        return fail(ctx, CTOX_UNSUPPORTED_OPERATION, "layer-stack models run on one GPU (the context has joined a group)");
    if (!c->vocab_size || !c->hidden_size || !c->num_layers || !c->kv_page_tokens || c->max_context_tokens < 2 * kMaxPass ||
        !(c->norm_eps >= 0.f) || !(c->logit_softcap >= 0.f))
        return fail(ctx, CTOX_SHAPE, "layer stack: sizes, page and context must be set");
    if (c->kv_dtype != CTOX_F32 && c->kv_dtype != CTOX_BF16)
        return fail(ctx, CTOX_UNSUPPORTED_DTYPE, "layer stack: kv dtype %u", c->kv_dtype);
    if (c->norm > CTOX_NORM_RMS || (c->out_norms && c->norm != CTOX_NORM_LAYER) || !std::isfinite(c->embed_scale))
        return fail(ctx, CTOX_UNSUPPORTED_OPERATION, "layer stack: norm %u (output norms %u), embedding scale %g", c->norm,
                    c->out_norms, (double)c->embed_scale);
    uint64_t mixed_values = 0;  // width of the values that layers mix
    for (uint32_t l = 0; l < c->num_layers; ++l) {
        const ctox_layer_config &y = layers[l];
        if (y.mixer < CTOX_MIXER_LATENT_ATTENTION || y.mixer > CTOX_MIXER_MATRIX_MEMORY)
            return fail(ctx, CTOX_UNSUPPORTED_OPERATION, "layer %u: unknown mixer %u", l, y.mixer);
        if (y.mlp > CTOX_MLP_CLAMPED_GLU)
            return fail(ctx, CTOX_UNSUPPORTED_OPERATION, "layer %u: unknown feed-forward %u", l, y.mlp);
        if ((y.mlp != CTOX_MLP_NONE && !y.ff) || (y.mlp == CTOX_MLP_CLAMPED_GLU && !(std::isfinite(y.mlp_limit) && std::isfinite(y.mlp_slope))))
            return fail(ctx, CTOX_SHAPE, "layer %u: unsupported feed-forward sizes", l);
        if (y.mixer != CTOX_MIXER_LATENT_ATTENTION && y.kv_from >= 0)
            return fail(ctx, CTOX_UNSUPPORTED_OPERATION, "layer %u: only latent attention reads another layer's cache", l);
        if (y.mixer == CTOX_MIXER_GROUPED_ATTENTION) {
            if (!y.heads || !y.kv_heads || y.heads % y.kv_heads || !y.dim || !y.vdim || y.rot_dim % 2 || y.rot_dim > y.dim ||
                !(y.rope_base > 0.0) || !std::isfinite(y.score_scale))
                return fail(ctx, CTOX_SHAPE, "layer %u: unsupported grouped-attention sizes", l);
            if (y.attn & CTOX_ATTN_V_MIX) {
                const uint64_t width = (uint64_t)y.kv_heads * y.vdim;
                if (mixed_values && mixed_values != width)
                    return fail(ctx, CTOX_SHAPE, "layer %u: mixes values of %llu with the first layer's of %llu", l,
                                (unsigned long long)width, (unsigned long long)mixed_values);
                mixed_values = width;
            }
            continue;
        }
        if (y.mixer == CTOX_MIXER_MATRIX_MEMORY) {
            if (!y.heads || !y.dim || !y.vdim || !(y.gate_cap > 0.f))
                return fail(ctx, CTOX_SHAPE, "layer %u: unsupported matrix-memory sizes", l);
            continue;
        }
        if (!y.heads || !y.dim || !y.vdim || !y.q_rank || !y.kv_rank || y.rot_dim % 2 || !(y.rope_base > 0.0) ||
            !std::isfinite(y.score_scale) || !(y.score_scale > 0.f))
            return fail(ctx, CTOX_SHAPE, "layer %u: unsupported latent-attention sizes", l);
        if (y.kv_from >= 0) {
            if ((uint32_t)y.kv_from >= l || layers[y.kv_from].kv_from >= 0 || layers[y.kv_from].mixer != y.mixer)
                return fail(ctx, CTOX_SHAPE, "layer %u: kv_from must name an earlier layer with its own cache", l);
            const ctox_layer_config &o = layers[y.kv_from];
            if (o.kv_rank != y.kv_rank || o.rot_dim != y.rot_dim || o.rope_base != y.rope_base)
                return fail(ctx, CTOX_SHAPE, "layer %u: latent and rotation differ from those of layer %d", l, y.kv_from);
        }
    }
    ctox_exec *e = new ctox_exec();
    StackModel *s = new StackModel();
    e->ctx = ctx;
    e->stack = s;
    s->c = *c;
    s->pass_cap = kDensePass;
    s->layers.resize(c->num_layers);
    bool first_values = false;
    for (uint32_t l = 0; l < c->num_layers; ++l) {
        StackLayer &L = s->layers[l];
        L.c = layers[l];
        const bool latent = L.c.mixer == CTOX_MIXER_LATENT_ATTENTION, grouped = L.c.mixer == CTOX_MIXER_GROUPED_ATTENTION;
        L.owner = latent && L.c.kv_from >= 0 ? (uint32_t)L.c.kv_from : l;
        L.dim_pad = round_up(L.c.dim, 16);
        L.vdim_pad = round_up(L.c.vdim, 16);
        if (latent) {
            L.rot_pad = round_up(L.c.rot_dim, 16);
            L.kv_pad = round_up(L.c.kv_rank, 16);
            L.slot_cols = L.kv_pad + L.rot_pad;
        } else if (grouped) {
            L.slot_cols = L.c.kv_heads * (L.dim_pad + L.vdim_pad);
            if (L.c.attn & CTOX_ATTN_V_MIX) {
                L.mixes_values = first_values;
                first_values = true;
            }
        } else {
            L.gate_row = round_up(2 * L.c.heads * (L.dim_pad + L.vdim_pad), 32);
        }
        L.head_w = L.dim_pad + L.rot_pad;
    }
    // Passes longer than kDensePass use the tensor-core products; in 32-bit mode, with pages that are not
    // whole tiles or with heads too large for its shared memory, every pass is a short one.
    bool longer = c->kv_dtype == CTOX_BF16 && c->kv_page_tokens % 128 == 0;
    for (const StackLayer &L : s->layers)
        longer = longer && (L.c.mixer == CTOX_MIXER_MATRIX_MEMORY ? memory_long_fits(ctx, memory_args(s, L))
                                                                 : prefill_attention_fits(ctx, L.dim_pad, L.rot_pad, L.vdim_pad));
    if (longer) s->pass_cap = std::max(kDensePass, std::min(c->pass_tokens ? c->pass_tokens : kDefaultPass, c->max_context_tokens));
    // what the executor's own calls read of the model
    e->cfg.vocab_size = c->vocab_size;
    e->cfg.hidden_size = c->hidden_size;
    e->cfg.num_hidden_layers = c->num_layers;
    e->cfg.max_context_tokens = c->max_context_tokens;
    e->cfg.kv_page_tokens = c->kv_page_tokens;
    e->cfg.kv_dtype = c->kv_dtype;
    e->n_layers = c->num_layers;
    e->vocab_l = c->vocab_size;
    *out = e;
    return CTOX_OK;
}

void stack_destroy(ctox_exec *e) {
    delete e->stack;
    e->stack = nullptr;
}

ctox_status stack_load_matrix(ctox_exec *e, uint32_t layer, uint32_t tensor, const ctox_fused_matvec_op *op) {
    ctox_ctx *ctx = e->ctx;
    CTOX_CUDA(ctx, cudaSetDevice(ctx->device));
    Placement p;
    if (!place(e, layer, tensor, &p))
        return fail(ctx, CTOX_INVALID_ARTIFACT, "tensor %u is not a matrix of layer %u", tensor, layer);
    if (op->rows != p.rows || op->columns != p.cols)
        return fail(ctx, CTOX_SHAPE, "tensor %u of layer %u is %llux%llu, expected %llux%llu", tensor, layer,
                    (unsigned long long)op->rows, (unsigned long long)op->columns, (unsigned long long)p.rows,
                    (unsigned long long)p.cols);
    if (op->dtype != CTOX_BF16 || op->weights_len != p.rows * p.cols * 2 || !op->weights)
        return fail(ctx, CTOX_UNSUPPORTED_DTYPE, "matrices of a layer stack are dense bf16 rows");
    if (op->activation != CTOX_ACT_IDENTITY || op->bias || op->s_in || op->s_out)
        return fail(ctx, CTOX_UNSUPPORTED_OPERATION, "matrices of a layer stack carry no bias, scales or activation");
    __nv_bfloat16 *tmp = nullptr;
    ctox_status rc = dev_alloc(ctx, (void **)&tmp, op->weights_len);
    if (rc) return rc;
    auto upload = [&]() -> ctox_status {
        CTOX_CUDA(ctx, cudaMemcpyAsync(tmp, op->weights, op->weights_len, cudaMemcpyHostToDevice, ctx->stream));
        for (int i = 0; i < p.n; ++i) {
            const Placement::To &t = p.to[i];
            EX(dense_alloc(e, t.mat, t.mat_rows, t.mat_cols));
            EX(launch_relayout(ctx, tmp, (uint32_t)p.rows, (uint32_t)p.cols, t.ra, t.ca,
                               t.mat->w + (size_t)t.row0 * t.mat->ld, t.mat->ld, t.transpose_group, t.transpose_cols));
        }
        CTOX_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
        return CTOX_OK;
    };
    rc = upload();
    dev_free(ctx, tmp, op->weights_len);
    if (rc) return rc;
    *p.loaded |= bit(tensor);
    e->warmed = false;
    return CTOX_OK;
}

bool stack_vector_slot(ctox_exec *e, uint32_t layer, uint32_t tensor, VectorSlot *slot) {
    StackModel *s = e->stack;
    slot->n = s->c.hidden_size;
    if (layer == CTOX_LAYER_GLOBAL) {
        slot->loaded = &s->loaded;
        slot->base = &s->final_norm;
        return tensor == CTOX_T_FINAL_NORM;
    }
    if (layer >= s->layers.size()) return false;
    StackLayer &L = s->layers[layer];
    const ctox_layer_config &c = L.c;
    const bool latent = c.mixer == CTOX_MIXER_LATENT_ATTENTION, grouped = c.mixer == CTOX_MIXER_GROUPED_ATTENTION,
               memory = c.mixer == CTOX_MIXER_MATRIX_MEMORY, mlp = c.mlp != CTOX_MLP_NONE, out = s->c.out_norms;
    slot->loaded = &L.loaded;
    auto at = [&](bool has, float **base, uint64_t n, uint64_t offset = 0, uint64_t total = 0) {
        slot->base = base;
        slot->n = n;
        slot->offset = offset;
        slot->total = total;
        return has;
    };
    const uint64_t H = s->c.hidden_size, nq = (uint64_t)c.heads * c.dim, nk = (uint64_t)c.kv_heads * c.dim,
                   nv = (uint64_t)c.kv_heads * c.vdim;
    const bool bias = grouped && (c.attn & CTOX_ATTN_BIAS), qk_norm = grouped && (c.attn & CTOX_ATTN_QK_NORM);
    switch (tensor) {
        case CTOX_T_INPUT_NORM: return at(true, &L.norm1, H);
        case CTOX_T_MIX_OUT_NORM: return at(out, &L.norm1b, H);
        case CTOX_T_POST_NORM: return at(mlp, &L.norm2, H);
        case CTOX_T_MLP_OUT_NORM: return at(mlp && out, &L.norm2b, H);
        case CTOX_T_Q_DOWN_NORM: return at(latent, &L.q_norm, c.q_rank);
        case CTOX_T_KV_DOWN_NORM: return at(latent && c.kv_from < 0, &L.kv_norm, c.kv_rank);
        case CTOX_T_Q_NORM: return at(qk_norm, &L.q_norm, nq);
        case CTOX_T_K_NORM: return at(qk_norm, &L.k_norm, nk);
        case CTOX_T_MIX_Q_BIAS: return at(bias, &L.fan_bias, nq, 0, nq + nk + nv);
        case CTOX_T_MIX_K_BIAS: return at(bias, &L.fan_bias, nk, nq, nq + nk + nv);
        case CTOX_T_MIX_V_BIAS: return at(bias, &L.fan_bias, nv, nq + nk, nq + nk + nv);
        case CTOX_T_MIX_O_BIAS: return at(bias, &L.o_bias, H);
        case CTOX_T_ATTN_SINK: return at(grouped && (c.attn & CTOX_ATTN_SINK), &L.sink, c.heads);
        case CTOX_T_V_MIX: return at(grouped && (c.attn & CTOX_ATTN_V_MIX), &L.v_mix, 1);
        case CTOX_T_MIX_HEAD_NORM: return at(memory, &L.head_norm, (uint64_t)c.heads * c.vdim);
        case CTOX_T_MEM_IN_BIAS: return at(memory, &L.in_bias, c.heads);
        case CTOX_T_MEM_FORGET_BIAS: return at(memory, &L.forget_bias, c.heads);
        default: return false;
    }
}

ctox_status stack_reset(ctox_exec *e) {
    StackModel *s = e->stack;
    if (s->memory) CTOX_CUDA(e->ctx, cudaMemsetAsync(s->memory, 0, s->memory_floats * 4, e->ctx->stream));
    return CTOX_OK;
}

ctox_status stack_fill_synthetic(ctox_exec *e, uint64_t seed) {
    ctox_ctx *ctx = e->ctx;
    StackModel *s = e->stack;
    uint64_t sd = seed * 1000003ull + 29;
    auto fill = [&](uint32_t layer, uint32_t tensor) -> ctox_status {
        Placement p;
        if (!place(e, layer, tensor, &p)) return CTOX_OK;
        for (int i = 0; i < p.n; ++i) {
            const Placement::To &t = p.to[i];
            EX(dense_alloc(e, t.mat, t.mat_rows, t.mat_cols));
            const uint64_t rows = t.fill_rows ? t.fill_rows : t.mat_rows;
            sd = sd * 6364136223846793005ull + 1442695040888963407ull;
            EX(launch_fill_normal_bf16(ctx, t.mat->w + (size_t)t.row0 * t.mat->ld, rows * t.mat->ld,
                                       1.0f / std::sqrt((float)p.cols), sd));
        }
        *p.loaded |= bit(tensor);
        return CTOX_OK;
    };
    auto constant = [&](uint32_t layer, uint32_t tensor, float value) -> ctox_status {
        VectorSlot slot;
        if (!stack_vector_slot(e, layer, tensor, &slot)) return CTOX_OK;
        const uint64_t total = slot.total ? slot.total : slot.n;
        if (!*slot.base) EX(xalloc(e, (void **)slot.base, total * 4, false));
        const std::vector<float> v(slot.n, value);
        CTOX_CUDA(ctx, cudaMemcpyAsync(*slot.base + slot.offset, v.data(), slot.n * 4, cudaMemcpyHostToDevice, ctx->stream));
        CTOX_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
        *slot.loaded |= bit(tensor);
        return CTOX_OK;
    };
    for (uint32_t t : {CTOX_T_EMBED, CTOX_T_LM_HEAD}) EX(fill(CTOX_LAYER_GLOBAL, t));
    EX(constant(CTOX_LAYER_GLOBAL, CTOX_T_FINAL_NORM, 1.f));
    for (uint32_t l = 0; l < s->layers.size(); ++l) {
        for (uint32_t t : {CTOX_T_Q_DOWN, CTOX_T_KV_DOWN, CTOX_T_Q_UP, CTOX_T_K_UP, CTOX_T_V_UP, CTOX_T_ATTN_O, CTOX_T_MIX_Q,
                           CTOX_T_MIX_K, CTOX_T_MIX_V, CTOX_T_MIX_GATE, CTOX_T_MEM_IN, CTOX_T_MEM_FORGET, CTOX_T_MLP_GATE,
                           CTOX_T_MLP_UP, CTOX_T_MLP_DOWN})
            EX(fill(l, t));
        for (uint32_t t : {CTOX_T_INPUT_NORM, CTOX_T_MIX_OUT_NORM, CTOX_T_POST_NORM, CTOX_T_MLP_OUT_NORM, CTOX_T_Q_DOWN_NORM,
                           CTOX_T_KV_DOWN_NORM, CTOX_T_Q_NORM, CTOX_T_K_NORM, CTOX_T_MIX_HEAD_NORM})
            EX(constant(l, t, 1.f));
        for (uint32_t t : {CTOX_T_MIX_Q_BIAS, CTOX_T_MIX_K_BIAS, CTOX_T_MIX_V_BIAS, CTOX_T_MIX_O_BIAS, CTOX_T_ATTN_SINK,
                           CTOX_T_MEM_IN_BIAS})
            EX(constant(l, t, 0.f));
        EX(constant(l, CTOX_T_V_MIX, 0.5f));
        EX(constant(l, CTOX_T_MEM_FORGET_BIAS, 3.f));  // a memory that lasts
    }
    CTOX_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
    e->warmed = false;
    return CTOX_OK;
}

namespace {

// Attention of a short pass, of either kind.
CacheAttn cache_args(const ctox_exec *e, const StackLayer &L, uint32_t m, uint32_t pos0) {
    const StackModel *s = e->stack;
    const StackLayer &O = s->layers[L.owner];
    CacheAttn a{};
    a.cache = O.cache;
    a.bf16 = s->c.kv_dtype == CTOX_BF16;
    a.page_table = O.page_table;
    a.page_tokens = s->c.kv_page_tokens;
    a.heads = L.c.heads;
    a.slot_cols = L.slot_cols;
    if (L.c.mixer == CTOX_MIXER_LATENT_ATTENTION) {
        a.q = s->q_abs;
        a.q_stride = a.q_cols = L.kv_pad;
        a.q_tail = s->q + L.dim_pad;
        a.tail_stride = L.head_w;
        a.kv_heads = 1;
        a.head_cols = a.key_cols = L.slot_cols;
        a.val_cols = L.kv_pad;
    } else {
        a.q = s->q;
        a.q_stride = a.q_cols = a.key_cols = a.val_off = L.dim_pad;
        a.kv_heads = L.c.kv_heads;
        a.head_cols = L.dim_pad + L.vdim_pad;
        a.val_cols = L.vdim_pad;
        a.out = s->att;
        a.sink = L.sink;
        a.arrived = s->arrived;
    }
    a.pos0 = pos0;
    a.m = m;
    a.window = L.c.window;
    a.scale = L.c.score_scale;
    a.ws_o = s->ws_o;
    a.ws_ml = s->ws_ml;
    return a;
}

}  // namespace

ctox_status stack_warmup(ctox_exec *e) {
    ctox_ctx *ctx = e->ctx;
    StackModel *s = e->stack;
    const ctox_stack_config &c = s->c;
    if ((s->loaded & global_needs(s)) != global_needs(s))
        return fail(ctx, CTOX_INVALID_STATE, "warmup: embedding, lm_head or final norm missing");
    for (uint32_t l = 0; l < s->layers.size(); ++l) {
        const uint64_t need = layer_needs(s, s->layers[l]);
        if ((s->layers[l].loaded & need) != need)
            return fail(ctx, CTOX_INVALID_STATE, "warmup: layer %u has missing tensors (mask %llx)", l,
                        (unsigned long long)(need & ~s->layers[l].loaded));
    }
    if (s->x[0]) return CTOX_OK;
    const uint64_t H = c.hidden_size, P = s->pass_cap, S = kDensePass;
    const bool longer = P > kDensePass;
    uint64_t fan_n = 0, q_w = 0, abs_w = 0, att_w = 0, ff = 1, ws_o = 0, ws_ml = 0, tiles = 0, first_w = 0;
    for (StackLayer &L : s->layers) {
        const bool memory = L.c.mixer == CTOX_MIXER_MATRIX_MEMORY;
        // a long pass keeps the projections of a matrix memory elsewhere
        fan_n = std::max<uint64_t>(fan_n, L.fan.rows * (memory ? S : P));
        att_w = std::max<uint64_t>(att_w, (uint64_t)L.c.heads * L.vdim_pad);
        ff = std::max<uint64_t>(ff, L.c.mlp != CTOX_MLP_NONE ? L.c.ff : 1);
        if (memory) {
            const MatrixMemory a = memory_args(s, L);
            s->memory_floats += a.heads * (memory_rows(a) * a.dim_pad + 4);
            continue;
        }
        q_w = std::max<uint64_t>(q_w, (uint64_t)L.c.heads * L.head_w);
        abs_w = std::max<uint64_t>(abs_w, (uint64_t)L.c.heads * L.kv_pad);
        if (L.c.attn & CTOX_ATTN_V_MIX) first_w = (uint64_t)L.c.kv_heads * L.c.vdim;
        for (uint32_t m = 1; m <= S; ++m) {
            CacheAttn a = cache_args(e, L, m, c.max_context_tokens);
            const uint64_t rows = (uint64_t)cache_attn_splits(ctx, a) * m * L.c.heads;
            ws_o = std::max<uint64_t>(ws_o, rows * a.val_cols);
            ws_ml = std::max<uint64_t>(ws_ml, rows * 2);
            tiles = std::max<uint64_t>(tiles, cache_attn_tiles(ctx, a));
        }
        const uint32_t pairs = std::max<uint32_t>(L.c.rot_dim / 2, 1);
        std::vector<float> freq(pairs, 0.f);
        for (uint32_t i = 0; i < L.c.rot_dim / 2; ++i)
            freq[i] = (float)std::pow(L.c.rope_base, -2.0 * (double)i / (double)L.c.rot_dim);
        EX(xalloc(e, (void **)&L.freq, pairs * 4, false));
        CTOX_CUDA(ctx, cudaMemcpyAsync(L.freq, freq.data(), pairs * 4, cudaMemcpyHostToDevice, ctx->stream));
        CTOX_CUDA(ctx, cudaStreamSynchronize(ctx->stream));  // `freq` is a local
    }
#define WALLOC(ptr, bytes)                                              \
    do {                                                                \
        const size_t bytes_ = (bytes);                                  \
        if (bytes_) EX(xalloc(e, (void **)&(ptr), bytes_, true));       \
    } while (0)
    if (longer) {
        uint64_t span = 0, k_w = 0, vt_w = 0, cq_w = 0, fan_b = 0, gates = 0;
        MemoryLongSizes mem{};
        for (uint32_t l = 0; l < s->layers.size(); ++l) {
            StackLayer &L = s->layers[l];
            if (L.c.mixer == CTOX_MIXER_MATRIX_MEMORY) {
                const MemoryLongSizes z = memory_long_sizes(memory_args(s, L), (uint32_t)P);
                mem.scan = std::max(mem.scan, z.scan);
                mem.delta = std::max(mem.delta, z.delta);
                mem.start = std::max(mem.start, z.start);
                mem.raw = std::max(mem.raw, z.raw);
                fan_b = std::max<uint64_t>(fan_b, L.gate_row);
                gates = std::max<uint64_t>(gates, 2ull * L.c.heads);
            }
            if (L.c.mixer != CTOX_MIXER_LATENT_ATTENTION) continue;
            const uint64_t reach = L.c.window ? L.c.window : c.max_context_tokens;
            span = std::max<uint64_t>(span, std::min<uint64_t>(reach + P, c.max_context_tokens));
            k_w = std::max<uint64_t>(k_w, (uint64_t)L.c.heads * L.dim_pad);
            vt_w = std::max<uint64_t>(vt_w, (uint64_t)L.c.heads * L.vdim_pad);
            cq_w = std::max<uint64_t>(cq_w, round_up(L.c.q_rank, 8));
            for (uint32_t other : s->table_layers)
                if (s->layers[other].c.rot_dim == L.c.rot_dim && s->layers[other].c.rope_base == L.c.rope_base)
                    L.table = s->layers[other].table;
            if (L.table || !L.c.rot_dim) continue;
            WALLOC(L.table, P * (L.c.rot_dim / 2) * sizeof(float2));
            s->table_layers.push_back(l);
        }
        s->span_cap = round_up((uint32_t)span, 128) + 128;
        WALLOC(s->h_b, P * round_up(c.hidden_size, 8) * 2);
        WALLOC(s->cq_b, P * cq_w * 2);
        WALLOC(s->q_b, P * q_w * 2);
        WALLOC(s->k_b, s->span_cap * k_w * 2);
        WALLOC(s->vt_b, s->span_cap * vt_w * 2);
        WALLOC(s->att_b, P * att_w * 2);
        WALLOC(s->u_b, P * round_up((uint32_t)ff, 8) * 2);
        WALLOC(s->head_b, (size_t)kHeadRowsLong * round_up(c.hidden_size, 8) * 2);
        WALLOC(s->fan_b, P * fan_b * 2);
        WALLOC(s->gates, P * gates * 4);
        WALLOC(s->mem_scan, mem.scan * 4);
        WALLOC(s->mem_delta, mem.delta * 4);
        WALLOC(s->mem_start, mem.start * 2);
        WALLOC(s->mem_raw, mem.raw * 4);
    }
    WALLOC(s->x[0], P * H * 4);
    WALLOC(s->x[1], P * H * 4);
    WALLOC(s->y, P * H * 4);
    WALLOC(s->fan, fan_n * 4);
    WALLOC(s->q, S * q_w * 4);
    WALLOC(s->q_abs, S * abs_w * 4);
    WALLOC(s->att, S * att_w * 4);
    WALLOC(s->u, S * ff * 4);
    WALLOC(s->ws_o, ws_o * 4);
    WALLOC(s->ws_ml, ws_ml * 4);
    WALLOC(s->arrived, tiles * 4);
    WALLOC(s->v_first, P * first_w * 4);
    WALLOC(s->rows_dev, P * 4);
    WALLOC(e->tokens_dev, (P + 1) * 4);
    WALLOC(e->hist_hidden, kMaxPass * H * 4);
    s->head_rows = longer ? kHeadRowsLong : (uint32_t)S;
    WALLOC(s->head_in, S * H * 4);
    WALLOC(e->logits, (size_t)s->head_rows * c.vocab_size * 4);
    WALLOC(s->memory, s->memory_floats * 4);
    uint64_t at = 0;
    for (StackLayer &L : s->layers) {
        if (L.c.mixer != CTOX_MIXER_MATRIX_MEMORY) continue;
        const MatrixMemory a = memory_args(s, L);
        L.state = s->memory + at;
        at += a.heads * memory_rows(a) * a.dim_pad;
        L.top = s->memory + at;
        at += a.heads * 4;  // keeps the next state on a 16-byte boundary
    }
    // caches: a ring of pages that holds the widest window read from it and one pass
    const uint32_t pt = c.kv_page_tokens, pages_total = (c.max_context_tokens + pt - 1) / pt;
    for (uint32_t l = 0; l < s->layers.size(); ++l) {
        StackLayer &O = s->layers[l];
        if (O.owner != l || !O.slot_cols) continue;
        uint64_t reach = 0;
        for (const StackLayer &L : s->layers)
            if (L.owner == l) reach = std::max<uint64_t>(reach, L.c.window ? L.c.window : c.max_context_tokens);
        const uint32_t ring = (uint32_t)std::min<uint64_t>(pages_total, (reach + P + pt - 1) / pt + 1);
        O.slots = ring * pt;
        WALLOC(O.cache, (size_t)O.slots * O.slot_cols * (c.kv_dtype == CTOX_BF16 ? 2 : 4));
        WALLOC(O.page_table, (size_t)pages_total * 4);
        std::vector<uint32_t> table(pages_total);
        for (uint32_t p = 0; p < pages_total; ++p) table[p] = p % ring;
        CTOX_CUDA(ctx, cudaMemcpyAsync(O.page_table, table.data(), (size_t)pages_total * 4, cudaMemcpyHostToDevice, ctx->stream));
        CTOX_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
    }
#undef WALLOC
    return CTOX_OK;
}

ctox_status stack_prefill_synthetic(ctox_exec *e, uint64_t n, uint64_t seed) {
    ctox_ctx *ctx = e->ctx;
    StackModel *s = e->stack;
    uint64_t sd = seed + 1;
    if (s->c.kv_dtype != CTOX_BF16)
        return fail(ctx, CTOX_UNSUPPORTED_OPERATION, "synthetic prefill of a layer stack needs a bf16 cache");
    for (StackLayer &L : s->layers) {
        if (!L.cache) continue;
        sd = sd * 6364136223846793005ull + 1442695040888963407ull;
        EX(launch_fill_normal_bf16(ctx, (__nv_bfloat16 *)L.cache, (uint64_t)L.slots * L.slot_cols, 1.f, sd));
    }
    if (s->memory) EX(launch_fill_normal_f32(ctx, s->memory, s->memory_floats, 0.02f, sd));
    (void)n;
    return CTOX_OK;
}

ctox_status stack_keep_streams(ctox_exec *e) {
    StackModel *s = e->stack;
    if (s->streams) return CTOX_OK;
    return xalloc(e, (void **)&s->streams,
                  (size_t)s->layers.size() * s->c.max_context_tokens * s->c.hidden_size * 4, true);
}

// ------------------------------------------------------------------ passes
namespace {

VecIn vec_plain(const float *x, uint32_t stride, uint32_t cols) {
    VecIn v{};
    v.x = x;
    v.x_stride = stride;
    v.cols = cols;
    return v;
}
VecOut vec_out(float *y, uint32_t stride, int kind = OUT_PLAIN) {
    VecOut o{};
    o.y = y;
    o.y_stride = stride;
    o.kind = kind;
    return o;
}

int stream_norm_kind(const StackModel *s) { return s->c.norm == CTOX_NORM_RMS ? NORM_RMS : NORM_LAYER; }

// The stream with the last sublayer's output added (normalised, if it has a norm), normalised by w: the
// prologue of the next product. The updated stream goes to the other buffer.
VecIn stream_in(StackModel *s, const float *w) {
    VecIn v = vec_plain(s->x[s->cur], s->c.hidden_size, s->c.hidden_size);
    v.norm = stream_norm_kind(s);
    v.w = w;
    v.eps = s->c.norm_eps;
    if (s->pending) {
        v.y = s->y;
        v.y_stride = s->c.hidden_size;
        v.wb = s->y_norm;
        v.x_out = s->x[s->cur ^ 1];
        s->cur ^= 1;
        s->pending = false;
    }
    return v;
}
// A sublayer has left its output in y.
void sublayer_done(StackModel *s, const float *out_norm) {
    s->pending = true;
    s->y_norm = out_norm;
}

LatentAppend append_args(const ctox_exec *e, const StackLayer &L, uint32_t pos0) {
    const StackModel *s = e->stack;
    return LatentAppend{s->fan, L.fan.rows, L.c.q_rank, L.c.kv_rank, L.c.rot_dim, L.kv_pad, L.rot_pad, L.kv_norm,
                        s->c.norm_eps, L.cache, s->c.kv_dtype == CTOX_BF16, L.page_table, s->c.kv_page_tokens, pos0,
                        L.freq};
}

// The mixers of up to kDensePass positions leave their output in y; the first product's prologue holds the
// residual add and the norm before the layer.
//
// Latent attention, six kernels: down projections, query up projection (norm in its prologue, rotation in its
// epilogue, cache append in its extra CTAs), queries into the latent space, attention, values (merge of the splits
// in the prologue), output projection.
ctox_status latent_short(ctox_exec *e, uint32_t l, uint32_t m, uint32_t pos0) {
    ctox_ctx *ctx = e->ctx;
    StackModel *s = e->stack;
    StackLayer &L = s->layers[l];
    const ctox_layer_config &c = L.c;
    const uint32_t H = s->c.hidden_size, qw = c.heads * L.head_w, vw = c.heads * L.vdim_pad;
    EX(launch_dense_matvec(ctx, L.fan, 1, m, stream_in(s, L.norm1), vec_out(s->fan, L.fan.rows), nullptr));
    VecIn in = vec_plain(s->fan, L.fan.rows, c.q_rank);
    in.norm = NORM_RMS;
    in.w = L.q_norm;
    in.eps = s->c.norm_eps;
    VecOut out = vec_out(s->q, qw, OUT_ROPE);
    out.head_width = L.head_w;
    out.rope0 = L.dim_pad;
    out.rope_dims = c.rot_dim;
    out.pos0 = pos0;
    out.freq = L.freq;
    const LatentAppend ap = append_args(e, L, pos0);
    EX(launch_dense_matvec(ctx, L.q_up, 1, m, in, out, L.owner == l ? &ap : nullptr));
    in = vec_plain(s->q, qw, L.dim_pad);
    in.x_group = L.head_w;
    EX(launch_dense_matvec(ctx, L.k_up_t, c.heads, m, in, vec_out(s->q_abs, c.heads * L.kv_pad), nullptr));
    const CacheAttn a = cache_args(e, L, m, pos0);
    const uint32_t splits = cache_attn_splits(ctx, a);
    EX(launch_cache_attention(ctx, a, splits));
    in = VecIn{};
    in.cols = L.kv_pad;
    in.ws_o = s->ws_o;
    in.ws_ml = s->ws_ml;
    in.splits = splits;
    in.ws_rows = m * c.heads;
    in.groups = c.heads;
    EX(launch_dense_matvec(ctx, L.v_up, c.heads, m, in, vec_out(s->att, vw), nullptr));
    return launch_dense_matvec(ctx, L.o, 1, m, vec_plain(s->att, vw, vw), vec_out(s->y, H), nullptr);
}

QkvPrep qkv_args(const ctox_exec *e, const StackLayer &L, uint32_t pos0) {
    const StackModel *s = e->stack;
    const ctox_layer_config &c = L.c;
    QkvPrep a{};
    a.fan = s->fan;
    a.fan_stride = L.fan.rows;
    a.heads = c.heads;
    a.kv_heads = c.kv_heads;
    a.dim = c.dim;
    a.vdim = c.vdim;
    a.dim_pad = L.dim_pad;
    a.vdim_pad = L.vdim_pad;
    a.rot_dim = c.rot_dim;
    a.q_norm = L.q_norm;
    a.k_norm = L.k_norm;
    a.eps = s->c.norm_eps;
    a.freq = L.freq;
    a.v_mix = L.mixes_values ? L.v_mix : nullptr;
    a.v_first = c.attn & CTOX_ATTN_V_MIX ? s->v_first : nullptr;
    a.cache = L.cache;
    a.bf16 = s->c.kv_dtype == CTOX_BF16;
    a.page_table = L.page_table;
    a.page_tokens = s->c.kv_page_tokens;
    a.pos0 = pos0;
    return a;
}

// Grouped attention, four kernels: projections with their biases, norms / rotation / value mixing / cache append,
// attention with the merge of its splits, output projection.
ctox_status grouped_short(ctox_exec *e, uint32_t l, uint32_t m, uint32_t pos0) {
    ctox_ctx *ctx = e->ctx;
    StackModel *s = e->stack;
    StackLayer &L = s->layers[l];
    const uint32_t vw = L.c.heads * L.vdim_pad;
    VecOut out = vec_out(s->fan, L.fan.rows);
    out.bias = L.fan_bias;
    EX(launch_dense_matvec(ctx, L.fan, 1, m, stream_in(s, L.norm1), out, nullptr));
    QkvPrep prep = qkv_args(e, L, pos0);
    prep.q_f32 = s->q;
    EX(launch_qkv_prep(ctx, prep, m));
    const CacheAttn a = cache_args(e, L, m, pos0);
    EX(launch_cache_attention(ctx, a, cache_attn_splits(ctx, a)));
    out = vec_out(s->y, s->c.hidden_size);
    out.bias = L.o_bias;
    return launch_dense_matvec(ctx, L.o, 1, m, vec_plain(s->att, vw, vw), out, nullptr);
}

// Matrix memory, three kernels: projections and gates, the recurrence with norm and output gate, output projection.
ctox_status memory_short(ctox_exec *e, uint32_t l, uint32_t m) {
    ctox_ctx *ctx = e->ctx;
    StackModel *s = e->stack;
    StackLayer &L = s->layers[l];
    const uint32_t vw = L.c.heads * L.vdim_pad;
    EX(launch_dense_matvec(ctx, L.fan, 1, m, stream_in(s, L.norm1), vec_out(s->fan, L.fan.rows), nullptr));
    EX(launch_matrix_memory(ctx, memory_args(s, L), s->fan, L.fan.rows, L.gate_row, m, s->att));
    return launch_dense_matvec(ctx, L.o, 1, m, vec_plain(s->att, vw, vw), vec_out(s->y, s->c.hidden_size), nullptr);
}

// One layer for up to kDensePass positions. The feed-forward is two kernels.
ctox_status layer_short(ctox_exec *e, uint32_t l, uint32_t m, uint32_t pos0) {
    ctox_ctx *ctx = e->ctx;
    StackModel *s = e->stack;
    StackLayer &L = s->layers[l];
    const ctox_layer_config &c = L.c;
    EX(c.mixer == CTOX_MIXER_LATENT_ATTENTION    ? latent_short(e, l, m, pos0)
       : c.mixer == CTOX_MIXER_GROUPED_ATTENTION ? grouped_short(e, l, m, pos0)
                                                 : memory_short(e, l, m));
    sublayer_done(s, L.norm1b);
    if (c.mlp == CTOX_MLP_NONE) return CTOX_OK;
    VecOut up = vec_out(s->u, c.ff, c.mlp == CTOX_MLP_RELU2 ? OUT_RELU2 : OUT_CLAMPED_GLU);
    up.cap = c.mlp_limit;
    up.slope = c.mlp_slope;
    EX(launch_dense_matvec(ctx, L.up, 1, m, stream_in(s, L.norm2), up, nullptr));
    EX(launch_dense_matvec(ctx, L.down, 1, m, vec_plain(s->u, c.ff, c.ff), vec_out(s->y, s->c.hidden_size), nullptr));
    sublayer_done(s, L.norm2b);
    return CTOX_OK;
}

GemmOperand rows_of(const __nv_bfloat16 *p, uint32_t rows, uint32_t cols, uint32_t ld) {
    return GemmOperand{p, rows, cols, ld, nullptr, 0, 0, 0};
}
GemmOperand weight_of(const DenseMat &w) { return rows_of(w.w, w.rows, w.cols, w.ld); }
GemmOut gemm_out(void *d, uint32_t ld, bool bf16, int kind = OUT_PLAIN) {
    GemmOut o{};
    o.d = d;
    o.ld = ld;
    o.bf16 = bf16;
    o.kind = kind;
    return o;
}

StreamNorm stream_norm(const StackModel *s, const float *w) {
    StreamNorm n{};
    n.x = s->x[s->cur];
    n.norm = stream_norm_kind(s);
    n.y = s->pending ? s->y : nullptr;
    n.wb = s->pending ? s->y_norm : nullptr;
    n.w = w;
    n.eps = s->c.norm_eps;
    n.width = s->c.hidden_size;
    return n;
}

PrefillAttn prefill_args(const ctox_exec *e, const StackLayer &L, uint32_t m, uint32_t pos0) {
    const StackModel *s = e->stack;
    const StackLayer &O = s->layers[L.owner];
    const ctox_layer_config &c = L.c;
    const uint32_t first = c.window && pos0 + 1 > c.window ? pos0 + 1 - c.window : 0;
    PrefillAttn a{};
    a.row0 = first / 128 * 128;
    a.span = pos0 + m - a.row0;
    a.q = s->q_b;
    a.cache = (const __nv_bfloat16 *)O.cache;
    a.out = s->att_b;
    a.page_table = O.page_table;
    a.page_tokens = s->c.kv_page_tokens;
    a.slots = O.slots;
    a.heads = c.heads;
    a.dim_pad = L.dim_pad;
    a.vdim_pad = L.vdim_pad;
    a.slot_cols = L.slot_cols;
    a.pos0 = pos0;
    a.m = m;
    a.window = c.window;
    a.scale = c.score_scale;
    return a;
}

// The mixers of a long pass: products on the tensor cores over bf16 activations. h is the normalised stream.
//
// Latent attention: keys and values of the visible span are expanded from the cache.
ctox_status latent_long(ctox_exec *e, uint32_t l, const GemmOperand &h, uint32_t m, uint32_t pos0) {
    ctox_ctx *ctx = e->ctx;
    StackModel *s = e->stack;
    StackLayer &L = s->layers[l];
    const StackLayer &O = s->layers[L.owner];
    const ctox_layer_config &c = L.c;
    const uint32_t H = s->c.hidden_size, qw = c.heads * L.head_w, vw = c.heads * L.vdim_pad, cq_ld = round_up(c.q_rank, 8);
    EX(launch_gemm(ctx, h, weight_of(L.fan), gemm_out(s->fan, L.fan.rows, false)));
    const LatentAppend ap = append_args(e, L, pos0);
    EX(launch_latent_split(ctx, s->fan, L.fan.rows, c.q_rank, L.q_norm, s->c.norm_eps, s->cq_b, cq_ld,
                           L.owner == l ? &ap : nullptr, m));
    GemmOut q = gemm_out(s->q_b, qw, true, c.rot_dim ? OUT_ROPE : OUT_PLAIN);
    q.head_width = L.head_w;
    q.rope0 = L.dim_pad;
    q.rope_dims = c.rot_dim;
    q.table = L.table;
    EX(launch_gemm(ctx, rows_of(s->cq_b, m, c.q_rank, cq_ld), weight_of(L.q_up), q));
    PrefillAttn a = prefill_args(e, L, m, pos0);
    GemmOperand latents = rows_of((const __nv_bfloat16 *)O.cache, a.span, L.kv_pad, L.slot_cols);
    latents.page_table = O.page_table;
    latents.page_tokens = s->c.kv_page_tokens;
    latents.row0 = a.row0;
    latents.store_rows = O.slots;
    EX(launch_gemm(ctx, latents, weight_of(L.k_up), gemm_out(s->k_b, c.heads * L.dim_pad, true)));
    EX(launch_gemm(ctx, weight_of(L.v_up), latents, gemm_out(s->vt_b, s->span_cap, true)));
    a.k = s->k_b;
    a.vt = s->vt_b;
    a.vt_ld = s->span_cap;
    a.rot_pad = L.rot_pad;
    a.rot_off = L.kv_pad;
    EX(launch_prefill_attention(ctx, a));
    return launch_gemm(ctx, rows_of(s->att_b, m, vw, vw), weight_of(L.o), gemm_out(s->y, H, false));
}

// Grouped attention: keys and values are read from the cache as they are.
ctox_status grouped_long(ctox_exec *e, uint32_t l, const GemmOperand &h, uint32_t m, uint32_t pos0) {
    ctox_ctx *ctx = e->ctx;
    StackModel *s = e->stack;
    StackLayer &L = s->layers[l];
    const uint32_t vw = L.c.heads * L.vdim_pad;
    GemmOut out = gemm_out(s->fan, L.fan.rows, false);
    out.bias = L.fan_bias;
    EX(launch_gemm(ctx, h, weight_of(L.fan), out));
    QkvPrep prep = qkv_args(e, L, pos0);
    prep.q_b16 = s->q_b;
    EX(launch_qkv_prep(ctx, prep, m));
    PrefillAttn a = prefill_args(e, L, m, pos0);
    a.kv_heads = L.c.kv_heads;
    a.sink = L.sink;
    EX(launch_prefill_attention(ctx, a));
    out = gemm_out(s->y, s->c.hidden_size, false);
    out.bias = L.o_bias;
    return launch_gemm(ctx, rows_of(s->att_b, m, vw, vw), weight_of(L.o), out);
}

// Matrix memory: the projections as bf16, the gates' preactivations as fp32, the recurrence by chunks.
ctox_status memory_long(ctox_exec *e, uint32_t l, const GemmOperand &h, uint32_t m) {
    ctox_ctx *ctx = e->ctx;
    StackModel *s = e->stack;
    StackLayer &L = s->layers[l];
    const uint32_t vw = L.c.heads * L.vdim_pad;
    GemmOut out = gemm_out(s->fan_b, L.gate_row, true);
    out.split = L.gate_row;
    out.d2 = s->gates;
    out.ld2 = 2 * L.c.heads;
    EX(launch_gemm(ctx, h, weight_of(L.fan), out));
    const MemoryLong w{s->fan_b, L.gate_row, s->gates, s->att_b, s->mem_scan, s->mem_delta, s->mem_start, s->mem_raw};
    EX(launch_matrix_memory_long(ctx, memory_args(s, L), w, m));
    return launch_gemm(ctx, rows_of(s->att_b, m, vw, vw), weight_of(L.o), gemm_out(s->y, s->c.hidden_size, false));
}

ctox_status layer_long(ctox_exec *e, uint32_t l, uint32_t m, uint32_t pos0) {
    ctox_ctx *ctx = e->ctx;
    StackModel *s = e->stack;
    StackLayer &L = s->layers[l];
    const ctox_layer_config &c = L.c;
    const uint32_t H = s->c.hidden_size, h_ld = round_up(H, 8), ff_ld = round_up(c.ff, 8);
    auto norm_into_h = [&](const float *w) -> ctox_status {  // the stream in place, its norm as bf16
        StreamNorm n = stream_norm(s, w);
        n.x_out = n.y ? s->x[s->cur] : nullptr;
        n.bf16_out = s->h_b;
        n.bf16_ld = h_ld;
        s->pending = false;
        return launch_stream_norm(ctx, n, m);
    };
    EX(norm_into_h(L.norm1));
    const GemmOperand h = rows_of(s->h_b, m, H, h_ld);
    EX(c.mixer == CTOX_MIXER_LATENT_ATTENTION    ? latent_long(e, l, h, m, pos0)
       : c.mixer == CTOX_MIXER_GROUPED_ATTENTION ? grouped_long(e, l, h, m, pos0)
                                                 : memory_long(e, l, h, m));
    sublayer_done(s, L.norm1b);
    if (c.mlp == CTOX_MLP_NONE) return CTOX_OK;
    EX(norm_into_h(L.norm2));
    GemmOut up = gemm_out(s->u_b, ff_ld, true, c.mlp == CTOX_MLP_RELU2 ? OUT_RELU2 : OUT_CLAMPED_GLU);
    up.cap = c.mlp_limit;
    up.slope = c.mlp_slope;
    EX(launch_gemm(ctx, h, weight_of(L.up), up));
    EX(launch_gemm(ctx, rows_of(s->u_b, m, c.ff, ff_ld), weight_of(L.down), gemm_out(s->y, H, false)));
    sublayer_done(s, L.norm2b);
    return CTOX_OK;
}

}  // namespace

ctox_status stack_pass(ctox_exec *e, uint32_t m, uint64_t pos0) {
    ctox_ctx *ctx = e->ctx;
    StackModel *s = e->stack;
    const uint32_t H = s->c.hidden_size;
    s->cur = 0;
    s->pending = false;
    EX(launch_embed_dense(ctx, s->embed.w, s->embed.ld, e->tokens_dev, H, m, s->c.embed_scale, s->x[0]));
    if (m > kDensePass)
        for (uint32_t l : s->table_layers) {
            const StackLayer &L = s->layers[l];
            EX(launch_rope_table(ctx, L.freq, L.c.rot_dim / 2, (uint32_t)pos0, m, L.table));
        }
    for (uint32_t l = 0; l < s->layers.size(); ++l) {
        EX(m > kDensePass ? layer_long(e, l, m, (uint32_t)pos0) : layer_short(e, l, m, (uint32_t)pos0));
        if (s->streams) {  // evidence: the stream after this layer
            StreamNorm n = stream_norm(s, nullptr);
            n.x_out = s->streams + ((size_t)l * s->c.max_context_tokens + pos0) * H;
            EX(launch_stream_norm(ctx, n, m));
        }
    }
    StreamNorm n = stream_norm(s, s->final_norm);
    n.x += (size_t)(m - 1) * H;
    if (n.y) n.y += (size_t)(m - 1) * H;
    n.f32_out = e->hist_hidden;
    return launch_stream_norm(ctx, n, 1);
}

ctox_status stack_head_last(ctox_exec *e) {
    StackModel *s = e->stack;
    VecOut out = vec_out(e->logits, s->c.vocab_size, s->c.logit_softcap > 0.f ? OUT_SOFTCAP : OUT_PLAIN);
    out.cap = s->c.logit_softcap;
    return launch_dense_matvec(e->ctx, head_of(s), 1, 1, vec_plain(e->hist_hidden, s->c.hidden_size, s->c.hidden_size), out,
                               nullptr);
}

ctox_status stack_head_rows(ctox_exec *e, const uint32_t *rows, uint32_t n) {
    ctox_ctx *ctx = e->ctx;
    StackModel *s = e->stack;
    const uint32_t H = s->c.hidden_size;
    CTOX_CUDA(ctx, cudaMemcpyAsync(s->rows_dev, rows, n * 4, cudaMemcpyHostToDevice, ctx->stream));
    StreamNorm a = stream_norm(s, s->final_norm);
    a.rows = s->rows_dev;
    if (n > kDensePass) {
        a.bf16_out = s->head_b;
        a.bf16_ld = round_up(H, 8);
        EX(launch_stream_norm(ctx, a, n));
        GemmOut o = gemm_out(e->logits, s->c.vocab_size, false, s->c.logit_softcap > 0.f ? OUT_SOFTCAP : OUT_PLAIN);
        o.cap = s->c.logit_softcap;
        return launch_gemm(ctx, rows_of(s->head_b, n, H, a.bf16_ld), weight_of(head_of(s)), o);
    }
    a.f32_out = s->head_in;
    EX(launch_stream_norm(ctx, a, n));
    VecOut out = vec_out(e->logits, s->c.vocab_size, s->c.logit_softcap > 0.f ? OUT_SOFTCAP : OUT_PLAIN);
    out.cap = s->c.logit_softcap;
    return launch_dense_matvec(ctx, head_of(s), 1, n, vec_plain(s->head_in, H, H), out, nullptr);
}

}  // namespace ctox
