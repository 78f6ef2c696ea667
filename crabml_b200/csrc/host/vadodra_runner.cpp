// vadodra_runner.cpp -- host driver of the Vadodra decoder family over the C ABI (crabml_cuda.h + crabml_seqops.h).  Like the other runners it
// contains no arithmetic: it owns the weights' handles, says what a sequence holds (key and value rings per window-attention layer, a ring of
// latent cache rows per latent-attention layer that has a cache of its own) and in which order the tensor ops run.  Slots, step and greedy
// generation are the shared ones of seq_runner.hpp, latent attention is the one of mixers.hpp.
//
//   layer:   ONE product of everything that multiplies the normed input, the norm inside it ; the mixer up to its heads' outputs ;
//            x += ONE product of the stacked output projections over [heads' outputs | gated units], the units and the sum inside it
//   window:  (q, k norms), rotation, keys and raw keys (the values) into the rings, one kernel ; masked softmax
//   latent:  attention over the ring of this layer or of the one it shares, times a gate per head
#include <string>
#include <vector>

#include "../../../include/crabml_vadodra.h"
#include "mixers.hpp"

using crabml::CudaTensor;
using crabml::TensorError;

namespace {

struct Layer {
    cvd_layer_config c{};
    CudaTensor norm, h_stack, o_stack, q_norm, k_norm, rot_freq;
    crabml::LatentAttention att;
    int64_t k_col = 0, g_col = 0, kv_col = 0, gate_col = 0;      // first columns of the stacked product's blocks (q starts at 0; up follows gate)
    int64_t ring = 0;                                            // rows of the layer's own ring(s)
    bool whole = false;                                          // window: the rings hold the whole sequence, no row is overwritten
};
struct LayerState {
    CudaTensor kring, vring;                                     // window; latent with a cache of its own: kring only
};
struct State : crabml::SeqState {
    std::vector<LayerState> layers;
};

struct Runner : csr_runner {
    cvd_config conf{};
    std::vector<Layer> layers;
    CudaTensor embed, final_norm, head;

    std::unique_ptr<crabml::SeqState> make_state() override {
        auto s = std::make_unique<State>();
        for (const Layer& L : layers) {
            LayerState st;
            if (L.c.mixer == CVD_MIXER_WINDOW) {
                st.kring = CudaTensor::alloc({L.ring, (int64_t)L.c.kv_heads * L.c.dim}, CC_F32, dev);
                st.vring = CudaTensor::alloc({L.ring, (int64_t)L.c.kv_heads * L.c.dim}, CC_F32, dev);
            } else if (L.c.kv_from < 0) {
                st.kring = CudaTensor::alloc({L.ring, L.att.row()}, CC_F32, dev);
            }
            s->layers.push_back(std::move(st));
        }
        return s;
    }
    // nothing to reset: a query at position i only reads rows of positions <= i of ITS sequence, all written since the slot was opened
    void reset_state(crabml::SeqState&) override {}

    CudaTensor norm_product(const CudaTensor& x, const CudaTensor& norm, const CudaTensor& w) {
        cc_view xv = x.view(), nv = norm.view(), wv = w.view();
        cc_buf* b = nullptr;
        check(cc_layer_norm_product(dev, &xv, &nv, nullptr, conf.norm_eps, &wv, &b));
        return adopt(b, {x.shape()[0], w.shape()[0]});
    }
    CudaTensor window_mixer(const Layer& L, LayerState& st, const CudaTensor& all, int64_t pos0) {
        const auto& c = L.c;
        const int64_t n = all.shape()[0];
        if (L.whole && pos0 + n > L.ring)
            throw TensorError("a sequence of " + std::to_string(pos0 + n) + " tokens does not fit the cache of " + std::to_string(L.ring));
        cc_view av = all.view(), kr = st.kring.view(), vr = st.vring.view(), qw = L.q_norm.view(), kw = L.k_norm.view(), fr{};
        cc_buf* b = nullptr;
        check(cc_qk_prepare_append_cols(dev, &av, 0, (int32_t)L.k_col, (int32_t)L.k_col, &kr, &vr, CC_QK_NORM_HEAD, &qw, &kw, conf.norm_eps, crabml::opt_view(L.rot_freq, fr),
                                        CC_ROPE_NEIGHBOURS, 0, c.rot_mag, pos0, c.heads, c.kv_heads, c.dim, c.dim, &b));
        CudaTensor q = adopt(b, {n, (int64_t)c.heads * c.dim});
        cc_view qv = q.view();
        b = nullptr;
        check(cc_masked_attention(dev, &qv, &kr, &vr, pos0, c.heads, c.kv_heads, c.dim, c.dim, c.window, 0, c.scale, nullptr, &b));
        return adopt(b, {n, (int64_t)c.heads * c.dim});
    }
    CudaTensor latent_mixer(size_t li, State& s, const CudaTensor& all, int64_t pos0) {
        const Layer& L = layers[li];
        const bool own = L.c.kv_from < 0;
        CudaTensor& ring = s.layers[own ? li : (size_t)L.c.kv_from].kring;
        if (L.att.few_rows(all.shape()[0])) return L.att.attend_few(*this, ring, all, 0, own ? &all : nullptr, L.kv_col, &all, L.g_col, pos0);
        CudaTensor y = L.att.attend_rotated(*this, ring, L.att.prepare_many(*this, ring, all, 0, own ? L.kv_col : -1, pos0), pos0);
        cc_view yv = y.view(), av = all.view();
        check(cc_head_gate_cols(dev, &yv, &av, (int32_t)L.g_col, L.c.heads, CC_ACT_SIGMOID));
        return y;
    }

    CudaTensor forward_chunk(crabml::SeqState& base, int64_t pos0, const int64_t* tokens, int64_t n, int device_slot) override {
        State& s = static_cast<State&>(base);
        CudaTensor x = CudaTensor::alloc({n, conf.width}, CC_F32, dev);
        if (device_slot >= 0) x.copy_rows_from_slot(embed, device_slot);
        else x.copy_rows_from(embed, std::vector<int64_t>(tokens, tokens + n));
        for (size_t li = 0; li < layers.size(); li++) {
            const Layer& L = layers[li];
            CudaTensor all = norm_product(x, L.norm, L.h_stack);
            CudaTensor y = L.c.mixer == CVD_MIXER_WINDOW ? window_mixer(L, s.layers[li], all, pos0) : latent_mixer(li, s, all, pos0);
            cc_view xv = x.view(), ov = L.o_stack.view(), yv = y.view(), av = all.view();
            check(cc_joined_product_accumulate(dev, &xv, &ov, &yv, &av, (int32_t)L.gate_col, (int32_t)(L.gate_col + L.c.ff), L.c.ff, &L.c.glu));
            x = std::move(x).with_name("layer:" + std::to_string(li) + ":" + std::to_string(pos0));
        }
        return x;
    }

    CudaTensor logits_of(const CudaTensor& x, const std::vector<int64_t>& rows) override {
        bool all = (int64_t)rows.size() == x.shape()[0];
        for (size_t i = 0; all && i < rows.size(); i++) all = rows[i] == (int64_t)i;
        if (all) return norm_product(x, final_norm, head);                       // every row in order (a decoded token): no copy
        CudaTensor xs = CudaTensor::alloc({(int64_t)rows.size(), conf.width}, CC_F32, dev);
        xs.copy_rows_from(x, rows);
        return norm_product(xs, final_norm, head);
    }
};

}  // namespace

extern "C" CC_API int cvd_runner_create(cc_device* dev, const cvd_config* conf, const cvd_layer_config* lc, const cvd_layer_weights* lw, cc_buf* embed, cc_buf* final_norm,
                                        cc_buf* head, csr_runner** out) {
    if (!dev || !conf || !lc || !lw || !embed || !final_norm || !head || !out) return CC_ERR_ARG;
    Runner* r = new Runner();
    r->dev = dev;
    r->conf = *conf;
    if (r->conf.chunk <= 0) r->conf.chunk = 256;
    if (r->conf.max_seq <= 0) r->conf.max_seq = 4096;
    r->width = conf->width; r->vocab = conf->vocab; r->chunk = r->conf.chunk;
    std::string err;
    int rc = crabml::seq_guarded(r, &err, [&] {
        const int64_t D = conf->width;
        if (conf->n_layers < 1 || D < 1 || conf->vocab < 1) throw TensorError("bad model sizes");
        r->embed = CudaTensor::wrap(dev, embed, {conf->vocab, D});
        r->final_norm = CudaTensor::wrap(dev, final_norm, {D});
        r->head = CudaTensor::wrap(dev, head, {conf->vocab, D});
        r->layers.resize(conf->n_layers);
        for (int i = 0; i < conf->n_layers; i++) {
            Layer& L = r->layers[i];
            const cvd_layer_config& c = L.c = lc[i];
            const cvd_layer_weights& w = lw[i];
            const std::string at = "layer " + std::to_string(i) + ": ";
            auto need = [&](cc_buf* b, const char* name, std::vector<int64_t> shape) {
                if (!b) throw TensorError(at + "tensor '" + name + "' is missing");
                return CudaTensor::wrap(dev, b, shape);
            };
            if (c.heads < 1 || c.dim < 1 || c.vdim < 1 || c.ff < 0) throw TensorError(at + "bad head counts / sizes");
            L.norm = need(w.norm, "norm1", {D});
            const int64_t budget = std::max<int64_t>(r->conf.max_seq, r->conf.chunk);
            if (c.mixer == CVD_MIXER_WINDOW) {
                if (c.kv_heads < 1 || c.heads % c.kv_heads || c.vdim != c.dim) throw TensorError(at + "bad head counts / sizes of the window attention");
                L.q_norm = need(w.q_norm, "mix.q.norm", {c.dim}); L.k_norm = need(w.k_norm, "mix.k.norm", {c.dim});
                if (w.rot_freq) {
                    const int64_t pairs = cc_tensor_capacity(w.rot_freq);
                    if (2 * pairs > c.dim) throw TensorError(at + "more rotated pairs than a head holds");
                    L.rot_freq = CudaTensor::wrap(dev, w.rot_freq, {pairs});
                }
                L.k_col = (int64_t)c.heads * c.dim;
                L.gate_col = L.k_col + (int64_t)c.kv_heads * c.dim;
                // what the window lets the first token of a pass see, plus the pass; the longest sequence when the window reaches that far
                L.whole = c.window <= 0 || c.window >= budget;
                L.ring = L.whole ? budget : (int64_t)c.window - 1 + r->conf.chunk;
                r->state_bytes_per_slot += 2 * L.ring * c.kv_heads * c.dim * 4;
            } else if (c.mixer == CVD_MIXER_LATENT) {
                if (c.rot_dim < 0 || c.kv_rank < 1) throw TensorError(at + "bad sizes of the latent attention");
                crabml::LatentAttention& a = L.att;
                a.heads = c.heads; a.dim = c.dim; a.rot_dim = c.rot_dim; a.vdim = c.vdim; a.kv_rank = c.kv_rank; a.scale = c.scale; a.rot_mag = c.rot_mag; a.norm_eps = conf->norm_eps;
                a.pairing = CC_ROPE_HALVES; a.gate_per_head = true;
                a.set_weights(dev, at, w.uk, w.uv, w.uk_t, w.uv_f32, w.dkv_norm, nullptr, w.rot_freq);
                L.g_col = a.q_cols();
                L.kv_col = L.g_col + c.heads;
                L.gate_col = L.kv_col + (c.kv_from < 0 ? a.row() : 0);
                if (c.kv_from < 0) {
                    if (!a.dkv_norm.valid()) throw TensorError(at + "tensor 'mix.dkv.norm' is missing");
                    L.ring = a.ring_rows(r->conf.chunk, r->conf.max_seq);
                    r->state_bytes_per_slot += L.ring * a.row() * 4;
                } else {
                    if (c.kv_from >= i || lc[c.kv_from].mixer != CVD_MIXER_LATENT || lc[c.kv_from].kv_from >= 0)
                        throw TensorError(at + "a shared cache belongs to an earlier latent-attention layer with a cache of its own");
                    if (lc[c.kv_from].kv_rank != c.kv_rank || lc[c.kv_from].rot_dim != c.rot_dim) throw TensorError(at + "the shared cache's rows have other sizes");
                }
            } else throw TensorError(at + "unknown mixer");
            L.h_stack = need(w.h_stack, "the stack of everything that multiplies the normed input", {L.gate_col + 2 * (int64_t)c.ff, D});
            L.o_stack = need(w.o_stack, "mix.o and mlp.down side by side", {D, (int64_t)c.heads * c.vdim + c.ff});
        }
    });
    if (rc != CC_OK) {
        crabml::seq_set_create_error(err);
        delete r;
        return rc;
    }
    *out = r;
    return CC_OK;
}
