// mixers.hpp -- mixers that more than one family's runner drives: latent attention over a ring of shared cache rows (Meresun, Papunex, Vadodra) and the
// state-space mixer (Vuzinex, Papunex).  Like the runners they hold weights' handles and say in which order the tensor ops run; sizes,
// weights and constants are filled in by the family, the sequence's state (a ring; a matrix and a convolution tail) is passed in.
#pragma once

#include <cmath>
#include <string>
#include <vector>

#include "../../../include/crabml_seqops.h"
#include "seq_runner.hpp"

namespace crabml {

inline const cc_view* opt_view(const CudaTensor& t, cc_view& store) {
    if (!t.valid()) return nullptr;
    store = t.view();
    return &store;
}
// the column blocks of a stacked product as contiguous tensors
inline std::vector<CudaTensor> split_columns(csr_runner& r, const CudaTensor& all, const std::vector<int32_t>& widths) {
    cc_view av = all.view();
    std::vector<cc_buf*> outs(widths.size(), nullptr);
    r.check(cc_split_cols(r.dev, &av, (int32_t)widths.size(), widths.data(), outs.data()));
    std::vector<CudaTensor> part;
    for (size_t p = 0; p < outs.size(); p++) part.push_back(r.adopt(outs[p], {all.shape()[0], widths[p]}));
    return part;
}

// Latent attention: one cached row [c | r] per position (c: the normed key / value latent, r: a rotated key part all heads share), softmax with
// an optional sink and window.  Two forms of the same attention, chosen by the pass's row count:
//   few rows (decoding)  the key up-projection is folded into the queries, scores and sums run over the cached rows themselves, the value
//                        up-projection is applied to the result
//   many rows (prompts)  the cached rows are expanded into per-head keys and values with two dense products
struct LatentAttention {
    int32_t heads = 0, dim = 0, rot_dim = 0, vdim = 0, kv_rank = 0;
    int32_t window = 0;                                   // <= 0: every earlier position (the ring then holds the whole sequence)
    float scale = 1.0f, rot_mag = 1.0f, norm_eps = 0.0f;
    int32_t pairing = CC_ROPE_NEIGHBOURS;                 // which columns of the rotated part turn together
    bool gate_per_head = false;                           // few-row form with a gate: one number per head instead of one per output column
    CudaTensor dkv_norm, uk, uv, uk_t, uv_f32, sink, rot_freq;

    int64_t row() const { return (int64_t)kv_rank + rot_dim; }
    int64_t q_cols() const { return (int64_t)heads * (dim + rot_dim); }
    int64_t out_cols() const { return (int64_t)heads * vdim; }
    bool few_rows(int64_t n) const { return n * heads <= 64; }
    // rows of the ring: the window's reach behind the first token of a pass, plus the pass; without a window the longest sequence
    int64_t ring_rows(int64_t chunk, int64_t max_seq) const { return window > 0 ? (int64_t)window - 1 + chunk : std::max(max_seq, chunk); }

    // weights by role; `at` names the layer in errors.  dkv_norm is left out by a layer that reads another layer's cache
    void set_weights(cc_device* dev, const std::string& at, cc_buf* uk_b, cc_buf* uv_b, cc_buf* uk_t_b, cc_buf* uv_f32_b, cc_buf* dkv_norm_b, cc_buf* sink_b, cc_buf* freq_b) {
        auto need = [&](cc_buf* b, const char* name, std::vector<int64_t> shape) {
            if (!b) throw TensorError(at + "tensor '" + name + "' is missing");
            return CudaTensor::wrap(dev, b, shape);
        };
        uk = need(uk_b, "mix.uk", {(int64_t)heads * dim, kv_rank}); uv = need(uv_b, "mix.uv", {out_cols(), kv_rank});
        uk_t = need(uk_t_b, "mix.uk (per head transposed)", {(int64_t)heads * kv_rank, dim}); uv_f32 = need(uv_f32_b, "mix.uv (F32)", {out_cols(), kv_rank});
        if (uk_t.dtype() != CC_F32 || uv_f32.dtype() != CC_F32) throw TensorError(at + "the folded forms of mix.uk / mix.uv must be F32: they enter the 32-bit scores and sums");
        if (dkv_norm_b) dkv_norm = CudaTensor::wrap(dev, dkv_norm_b, {kv_rank});
        if (sink_b) sink = CudaTensor::wrap(dev, sink_b, {heads});
        if (freq_b) {
            const int64_t pairs = cc_tensor_capacity(freq_b);
            if (2 * pairs > rot_dim) throw TensorError(at + "more rotated pairs than the rotated part holds");
            rot_freq = CudaTensor::wrap(dev, freq_b, {pairs});
        }
    }
    void check_capacity(const CudaTensor& ring, int64_t end) const {
        if (window <= 0 && end > ring.shape()[0])
            throw TensorError("a sequence of " + std::to_string(end) + " tokens does not fit the cache of " + std::to_string(ring.shape()[0]));
    }

    // few rows: queries in the columns q_col0 .. of q_src, raw cache rows of the same tokens in the columns kv_col0 .. of kv_src (kv_src NULL: the
    // ring's layer has written them already), gate numbers in the columns gate_col0 .. of gate_src (NULL: not gated).  -> [n, heads * vdim]
    CudaTensor attend_few(csr_runner& r, CudaTensor& ring, const CudaTensor& q_src, int64_t q_col0, const CudaTensor* kv_src, int64_t kv_col0, const CudaTensor* gate_src,
                          int64_t gate_col0, int64_t pos0) const {
        const int64_t n = q_src.shape()[0];
        check_capacity(ring, pos0 + n);
        cc_view qv = q_src.view(), ukv = uk_t.view(), rv = ring.view(), kv{}, fq{}, nw{}, sk{};
        if (kv_src) kv = kv_src->view();
        cc_buf* b = nullptr;
        r.check(cc_latent_query_append_paired(r.dev, &qv, (int32_t)q_col0, &ukv, heads, rot_dim, opt_view(rot_freq, fq), pairing, rot_mag, pos0, kv_src ? &kv : nullptr, (int32_t)kv_col0, &rv,
                                       opt_view(dkv_norm, nw), norm_eps, &b));
        CudaTensor ql = r.adopt(b, {n, (int64_t)heads * row()});
        cc_view qlv = ql.view();
        b = nullptr;
        // all heads read the one cached row per position; keys are whole rows, values their first kv_rank columns
        r.check(cc_window_attention_sink(r.dev, &qlv, nullptr, 0.0f, &rv, nullptr, pos0, heads, 1, (int32_t)row(), kv_rank, window, scale, nullptr, nullptr, opt_view(sink, sk), &b));
        CudaTensor ol = r.adopt(b, {n, (int64_t)heads * kv_rank});
        cc_view olv = ol.view(), uvv = uv_f32.view();
        b = nullptr;
        if (gate_src) {
            cc_view gv = gate_src->view();
            r.check((gate_per_head ? cc_head_project_head_gated : cc_head_project_gated)(r.dev, &olv, &uvv, heads, &gv, (int32_t)gate_col0, &b));
        } else {
            r.check(cc_head_project(r.dev, &olv, &uvv, heads, 0, nullptr, 1.0f, 0, &b));
        }
        return r.adopt(b, {n, out_cols()});
    }
    // the cache rows of new tokens out of their raw rows
    void append(csr_runner& r, CudaTensor& ring, const CudaTensor& ckv, int64_t pos0) const {
        check_capacity(ring, pos0 + ckv.shape()[0]);
        cc_view rv = ring.view(), cv = ckv.view(), nw{}, fq{};
        r.check(cc_latent_ring_append(r.dev, &rv, &cv, opt_view(dkv_norm, nw), norm_eps, kv_rank, opt_view(rot_freq, fq), rot_mag, pos0));
    }
    // many rows: the queries in the columns q_col0 .. of src, rotated, as a tensor of their own; with kv_col0 >= 0 the tokens' cache rows as well
    CudaTensor prepare_many(csr_runner& r, CudaTensor& ring, const CudaTensor& src, int64_t q_col0, int64_t kv_col0, int64_t pos0) const {
        check_capacity(ring, pos0 + src.shape()[0]);
        cc_view sv = src.view(), rv = ring.view(), fq{}, nw{};
        cc_buf* b = nullptr;
        r.check(cc_latent_prepare_append(r.dev, &sv, (int32_t)q_col0, heads, dim, rot_dim, opt_view(rot_freq, fq), pairing, rot_mag, pos0, kv_col0 >= 0 ? &sv : nullptr,
                                         kv_col0 >= 0 ? (int32_t)kv_col0 : 0, &rv, opt_view(dkv_norm, nw), norm_eps, &b));
        return r.adopt(b, {src.shape()[0], q_cols()});
    }
    // many rows, the tokens' cache rows already in the ring; q: their raw queries (rotated in place).  -> [n, heads * vdim]
    CudaTensor attend_many(csr_runner& r, CudaTensor& ring, const CudaTensor& q, int64_t pos0) const {
        cc_view qv = q.view(), fq{};
        if (rot_freq.valid())
            r.check((pairing == CC_ROPE_HALVES ? cc_rope_halves : cc_rope_pairs)(r.dev, &qv, heads, dim + rot_dim, dim, opt_view(rot_freq, fq), rot_mag, pos0));
        return attend_rotated(r, ring, q, pos0);
    }
    CudaTensor attend_rotated(csr_runner& r, CudaTensor& ring, const CudaTensor& q, int64_t pos0) const {
        const int64_t n = q.shape()[0], cap = ring.shape()[0];
        check_capacity(ring, pos0 + n);
        cc_view qv = q.view(), rv = ring.view(), sk{};
        // the expansion keeps the ring's row order (position p in row p % ring), so the attention reads it like the ring itself; rows no token
        // has written yet are never visible
        const int64_t rows = std::min<int64_t>(cap, pos0 + n);
        CudaTensor lat = CudaTensor(ring).with_strider(TensorStrider({rows, kv_rank}, {row(), 1})).contiguous();
        CudaTensor kp = uk.matmul_vec(lat), v = uv.matmul_vec(lat);
        cc_view kpv = kp.view(), vv = v.view();
        cc_buf* b = nullptr;
        r.check(cc_head_concat_shared(r.dev, &kpv, &rv, heads, kv_rank, rot_dim, &b));
        CudaTensor keys = r.adopt(b, {rows, q_cols()});
        cc_view kv = keys.view();
        b = nullptr;
        r.check(cc_window_attention_sink(r.dev, &qv, nullptr, 0.0f, &kv, &vv, pos0, heads, heads, dim + rot_dim, vdim, window, scale, nullptr, nullptr, opt_view(sink, sk), &b));
        return r.adopt(b, {n, out_cols()});
    }
};

// The state-space mixer (the SSD form of Mamba-2): one in-projection z | x B C | dt, a short causal convolution with bias and silu over x B C, the
// scan, the gate by silu(z) BEFORE an RMS norm in groups, the output projection.  Every op reads its block of the in-projection where it lies.
struct StateSpace {
    int32_t heads = 0, vdim = 0, state = 0, groups = 1, conv = 1, norm_groups = 1;
    float norm_eps = 0.0f;
    CudaTensor in, conv_w, conv_bias, dt_bias, a_log, d_skip, norm, o;

    int64_t inner() const { return (int64_t)heads * vdim; }
    int64_t conv_cols() const { return inner() + 2 * (int64_t)groups * state; }
    int64_t state_floats() const { return (int64_t)heads * state * vdim + (int64_t)(conv - 1) * conv_cols(); }
    CudaTensor make_matrix(cc_device* dev) const { return CudaTensor::alloc({heads, state, vdim}, CC_F32, dev); }
    CudaTensor make_tail(cc_device* dev) const { return conv > 1 ? CudaTensor::alloc({conv - 1, conv_cols()}, CC_F32, dev) : CudaTensor(); }

    void set_weights(cc_device* dev, const std::string& at, int64_t width, cc_buf* in_b, cc_buf* conv_b, cc_buf* conv_bias_b, cc_buf* dt_bias_b, cc_buf* a_log_b, cc_buf* d_b, cc_buf* norm_b,
                     cc_buf* o_b) {
        if (heads < 1 || vdim < 1 || state < 1 || groups < 1 || heads % groups || conv < 1) throw TensorError(at + "bad sizes of the state-space mixer");
        if (norm_groups < 1 || inner() % norm_groups) throw TensorError(at + "the norm's groups do not divide the inner width");
        auto need = [&](cc_buf* b, const char* name, std::vector<int64_t> shape) {
            if (!b) throw TensorError(at + "tensor '" + name + "' is missing");
            return CudaTensor::wrap(dev, b, shape);
        };
        in = need(in_b, "mix.in", {inner() + conv_cols() + heads, width});
        conv_w = need(conv_b, "mix.conv", {conv_cols(), conv});
        if (conv_bias_b) conv_bias = CudaTensor::wrap(dev, conv_bias_b, {conv_cols()});
        dt_bias = need(dt_bias_b, "mix.dt_bias", {heads}); a_log = need(a_log_b, "mix.A_log", {heads});
        if (d_b) d_skip = CudaTensor::wrap(dev, d_b, {heads});
        norm = need(norm_b, "mix.norm", {inner()}); o = need(o_b, "mix.o", {width, inner()});
    }

    CudaTensor run(csr_runner& r, CudaTensor& S, CudaTensor& tail, const CudaTensor& h) const {
        const int64_t n = h.shape()[0];
        CudaTensor all = in.matmul_vec(h);                                          // z | x B C | dt
        cc_view av = all.view(), cw = conv_w.view(), cb{}, tl{};
        cc_buf* b = nullptr;
        r.check(cc_short_conv_cols(r.dev, &av, (int32_t)inner(), &cw, opt_view(conv_bias, cb), opt_view(tail, tl), CC_ACT_SILU, &b));
        CudaTensor xbc = r.adopt(b, {n, conv_cols()});
        cc_view xv = xbc.view(), db = dt_bias.view(), al = a_log.view(), ds{}, sv = S.view();
        b = nullptr;
        r.check(cc_state_space_scan_cols(r.dev, &xv, &av, (int32_t)(inner() + conv_cols()), &db, &al, opt_view(d_skip, ds), &sv, heads, groups, state, vdim, &b));
        CudaTensor y = r.adopt(b, {n, inner()});
        CudaTensor z = CudaTensor(all).with_strider(TensorStrider({n, inner()}, {all.shape()[1], 1}));
        cc_view yv = y.view(), zv = z.view(), nw = norm.view();
        r.check(cc_gated_group_rms_norm(r.dev, &yv, &yv, &zv, &nw, norm_groups, norm_eps, CC_ACT_SILU));
        return o.matmul_vec(y);
    }
};

}  // namespace crabml
