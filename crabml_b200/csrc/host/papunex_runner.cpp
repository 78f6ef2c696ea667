// papunex_runner.cpp -- host driver of the Papunex decoder family over the C ABI (crabml_cuda.h + crabml_seqops.h).  Like the other runners it
// contains no arithmetic: it owns the weights' handles, says what a sequence holds (a ring of latent cache rows per attention layer that has a
// cache of its own; a state matrix and a convolution tail per state-space layer) and in which order the tensor ops run.  Slots, step and greedy
// generation are the shared ones of seq_runner.hpp, both mixers those of mixers.hpp.
//
//   layer:   x += norm1(mixer(x)) ; x += norm2(ff(x))
//   latent:  ONE product of the stacked projections q | gate | (raw cache row) ; attention over the ring of this layer or of the one it shares ;
//            gate ; W_o
//   ff:      dense: W_down relu(W_up x)^2.  routed: router (+ the shared expert's gate) -> slots ; the chosen experts and the shared expert's pieces
//            in one weighted sum
#include <string>
#include <vector>

#include "../../../include/crabml_papunex.h"
#include "mixers.hpp"

using crabml::CudaTensor;
using crabml::TensorError;

namespace {

struct Layer {
    cpr_layer_config c{};
    CudaTensor norm1, norm2, h_stack, o, up, down, router, shared_gate;
    crabml::LatentAttention att;
    crabml::StateSpace ss;
    std::vector<int32_t> widths;                   // column blocks of h_stack's product: q, gate, (cache row)
    int64_t ring = 0;                              // latent, own cache: rows of the ring
};
struct LayerState {
    CudaTensor ring, S, tail;
};
struct State : crabml::SeqState {
    std::vector<LayerState> layers;
};

struct Runner : csr_runner {
    cpr_config conf{};
    std::vector<Layer> layers;
    CudaTensor embed, final_norm, head;

    std::unique_ptr<crabml::SeqState> make_state() override {
        auto s = std::make_unique<State>();
        for (const Layer& L : layers) {
            LayerState st;
            if (L.c.mixer == CPR_MIXER_STATE_SPACE) {
                st.S = L.ss.make_matrix(dev);
                st.tail = L.ss.make_tail(dev);
            } else if (L.c.kv_from < 0) {
                st.ring = CudaTensor::alloc({L.ring, L.att.row()}, CC_F32, dev);
            }
            s->layers.push_back(std::move(st));
        }
        return s;
    }
    // a reused slot starts like a new one: recurrence and convolution see nothing before position 0.  The rings need no reset: a query at
    // position i only reads rows of positions <= i of ITS sequence, all written since the slot was opened.
    void reset_state(crabml::SeqState& base) override {
        for (LayerState& st : static_cast<State&>(base).layers)
            for (CudaTensor* t : {&st.S, &st.tail})
                if (t->valid()) { cc_view v = t->view(); check(cc_tensor_zero(dev, &v)); }
    }

    CudaTensor latent_mixer(size_t li, State& s, const CudaTensor& x, int64_t pos0) {
        const Layer& L = layers[li];
        const bool own = L.c.kv_from < 0;
        CudaTensor& ring = s.layers[own ? li : (size_t)L.c.kv_from].ring;
        CudaTensor all = L.h_stack.matmul_vec(x);
        const int64_t q_cols = L.widths[0], g_cols = L.widths[1];
        if (L.att.few_rows(x.shape()[0])) return L.o.matmul_vec(L.att.attend_few(*this, ring, all, 0, own ? &all : nullptr, q_cols + g_cols, &all, q_cols, pos0));
        std::vector<CudaTensor> part = crabml::split_columns(*this, all, L.widths);
        if (own) L.att.append(*this, ring, part[2], pos0);
        CudaTensor y = L.att.attend_many(*this, ring, part[0], pos0);
        cc_view yv = y.view(), gv = part[1].view();
        check(cc_gated_sum(dev, &yv, 0, &yv, &gv, nullptr, nullptr, nullptr, nullptr));
        return L.o.matmul_vec(y);
    }

    CudaTensor feed_forward(const Layer& L, const CudaTensor& x) {
        const auto& c = L.c;
        const int64_t n = x.shape()[0];
        cc_view xv = x.view(), uv = L.up.view(), dv = L.down.view();
        cc_buf* b = nullptr;
        if (c.ff_kind == CPR_FF_DENSE) {
            check(cc_feed_forward_act(dev, &xv, &uv, &dv, CC_ACT_RELU_SQUARED, &b));
            return adopt(b, {n, conf.width});
        }
        cc_view rw = L.router.view(), sg{};
        cc_buf *ids = nullptr, *wts = nullptr;
        const cc_route_params rp = {CC_ROUTE_SOFTMAX, c.top, 1, 1, 1, 1, 1e-20f, c.route_scale};
        check(cc_moe_route_shared(dev, &xv, &rw, nullptr, crabml::opt_view(L.shared_gate, sg), c.shared, &rp, &ids, &wts));
        CudaTensor tid = adopt(ids, {n, c.top + c.shared}), tw = adopt(wts, {n, c.top + c.shared});
        cc_view iv = tid.view(), wv = tw.view();
        check(cc_moe_experts_act(dev, &xv, &iv, &wv, &uv, &dv, c.experts + c.shared, c.ff, CC_ACT_RELU_SQUARED, &b));
        return adopt(b, {n, conf.width});
    }

    // x += norm(y) * w
    void add_normed(const CudaTensor& x, const CudaTensor& y, const CudaTensor& w) {
        cc_view xv = x.view(), yv = y.view(), wv = w.view();
        check(cc_rms_norm_gain(dev, &xv, &yv, &wv, conf.norm_eps, 1));
    }

    CudaTensor forward_chunk(crabml::SeqState& base, int64_t pos0, const int64_t* tokens, int64_t n, int device_slot) override {
        State& s = static_cast<State&>(base);
        CudaTensor x = CudaTensor::alloc({n, conf.width}, CC_F32, dev);
        if (device_slot >= 0) x.copy_rows_from_slot(embed, device_slot);
        else x.copy_rows_from(embed, std::vector<int64_t>(tokens, tokens + n));
        for (size_t li = 0; li < layers.size(); li++) {
            const Layer& L = layers[li];
            add_normed(x, L.c.mixer == CPR_MIXER_LATENT ? latent_mixer(li, s, x, pos0) : L.ss.run(*this, s.layers[li].S, s.layers[li].tail, x), L.norm1);
            if (L.c.ff_kind != CPR_FF_NONE) add_normed(x, feed_forward(L, x), L.norm2);
            x = std::move(x).with_name("layer:" + std::to_string(li) + ":" + std::to_string(pos0));
        }
        return x;
    }

    CudaTensor logits_of(const CudaTensor& x, const std::vector<int64_t>& rows) override {
        bool all = (int64_t)rows.size() == x.shape()[0];
        for (size_t i = 0; all && i < rows.size(); i++) all = rows[i] == (int64_t)i;
        CudaTensor xs = x;                                                      // every row in order (a decoded token): no copy
        if (!all) {
            xs = CudaTensor::alloc({(int64_t)rows.size(), conf.width}, CC_F32, dev);
            xs.copy_rows_from(x, rows);
        }
        CudaTensor h = CudaTensor::alloc(xs.shape(), CC_F32, dev);
        cc_view hv = h.view(), xv = xs.view(), wv = final_norm.view();
        check(cc_group_rms_norm(dev, &hv, &xv, &wv, 1, conf.norm_eps));
        CudaTensor lg = head.matmul_vec(h);
        if (conf.softcap > 0.0f) { cc_view lv = lg.view(); check(cc_softcap_inplace(dev, &lv, conf.softcap)); }
        return lg;
    }
};

}  // namespace

extern "C" CC_API int cpr_runner_create(cc_device* dev, const cpr_config* conf, const cpr_layer_config* lc, const cpr_layer_weights* lw, cc_buf* embed, cc_buf* final_norm,
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
            const cpr_layer_config& c = L.c = lc[i];
            const cpr_layer_weights& w = lw[i];
            const std::string at = "layer " + std::to_string(i) + ": ";
            auto need = [&](cc_buf* b, const char* name, std::vector<int64_t> shape) {
                if (!b) throw TensorError(at + "tensor '" + name + "' is missing");
                return CudaTensor::wrap(dev, b, shape);
            };
            L.norm1 = need(w.norm1, "norm1", {D});
            if (c.mixer == CPR_MIXER_LATENT) {
                if (c.heads < 1 || c.dim < 1 || c.rot_dim < 0 || c.vdim < 1 || c.kv_rank < 1) throw TensorError(at + "bad head counts / sizes");
                crabml::LatentAttention& a = L.att;
                a.heads = c.heads; a.dim = c.dim; a.rot_dim = c.rot_dim; a.vdim = c.vdim; a.kv_rank = c.kv_rank; a.scale = c.scale; a.rot_mag = c.rot_mag; a.norm_eps = conf->norm_eps;
                a.set_weights(dev, at, w.uk, w.uv, w.uk_t, w.uv_f32, w.dkv_norm, w.sink, w.rot_freq);
                L.widths = {(int32_t)a.q_cols(), (int32_t)a.out_cols()};
                if (c.kv_from < 0) {
                    if (!a.dkv_norm.valid()) throw TensorError(at + "tensor 'mix.dkv.norm' is missing");
                    L.widths.push_back((int32_t)a.row());
                    L.ring = a.ring_rows(r->conf.chunk, r->conf.max_seq);
                    r->state_bytes_per_slot += L.ring * a.row() * 4;
                } else {
                    if (c.kv_from >= i || lc[c.kv_from].mixer != CPR_MIXER_LATENT || lc[c.kv_from].kv_from >= 0)
                        throw TensorError(at + "a shared cache belongs to an earlier latent-attention layer with a cache of its own");
                    if (lc[c.kv_from].kv_rank != c.kv_rank || lc[c.kv_from].rot_dim != c.rot_dim) throw TensorError(at + "the shared cache's rows have other sizes");
                }
                int64_t on_x = 0;
                for (int32_t v : L.widths) on_x += v;
                L.h_stack = need(w.h_stack, "the stack of mix.q, mix.g, mix.dkv", {on_x, D});
                L.o = need(w.o, "mix.o", {D, a.out_cols()});
            } else if (c.mixer == CPR_MIXER_STATE_SPACE) {
                crabml::StateSpace& m = L.ss;
                m.heads = c.s_heads; m.vdim = c.s_vdim; m.state = c.s_state; m.groups = c.s_groups; m.conv = c.s_conv; m.norm_groups = c.s_norm_groups; m.norm_eps = conf->norm_eps;
                m.set_weights(dev, at, D, w.in, w.conv, w.conv_bias, w.dt_bias, w.a_log, w.d_skip, w.s_norm, w.s_o);
                r->state_bytes_per_slot += m.state_floats() * 4;
            } else throw TensorError(at + "unknown mixer");
            if (c.ff_kind == CPR_FF_NONE) continue;
            if (c.ff < 1) throw TensorError(at + "bad feed-forward width");
            L.norm2 = need(w.norm2, "norm2", {D});
            int64_t units = 1;
            if (c.ff_kind == CPR_FF_ROUTED) {
                if (c.experts < 1 || c.top < 1 || c.top > c.experts || c.shared < 0) throw TensorError(at + "bad router sizes");
                L.router = need(w.router, "mlp.router", {c.experts, D});
                if (w.shared_gate) L.shared_gate = CudaTensor::wrap(dev, w.shared_gate, {D});
                if (L.shared_gate.valid() && c.shared == 0) throw TensorError(at + "a gate for a shared expert the layer does not have");
                units = (int64_t)c.experts + c.shared;
            } else if (c.ff_kind != CPR_FF_DENSE) throw TensorError(at + "unknown feed-forward kind");
            L.up = need(w.up, "mlp up", {units * c.ff, D});
            L.down = need(w.down, "mlp down", {units * D, c.ff});
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
