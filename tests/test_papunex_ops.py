"""The mechanisms the Papunex family added to include/crabml_seqops.h or shares in another form, each alone, against its function in the plain
reference (tests/papunex_ref.py).  Where random inputs would hide a fault (a far key, a sink, a page of a pass) the inputs are made so that it
shows."""
import numpy as np
import pytest

from crabml_b200 import capi, rotary, seqops
from crabml_b200.safetensors import bf16_to_f32, f32_to_bf16
from tests import papunex_ref as R
from tests.gpu_common import make_device

pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module")
def dev():
    d = make_device()
    yield d
    d.close()


def T32(dev, a, shape=None):
    from crabml_b200 import CudaTensor
    a = np.asarray(a, np.float32)
    return CudaTensor.new(a, list(shape if shape is not None else a.shape), dev)


def W(dev, a, dtype):
    from crabml_b200 import CudaTensor
    a = np.ascontiguousarray(a, np.float32)
    if dtype == capi.BF16:
        return CudaTensor.from_cpu(f32_to_bf16(a).reshape(a.shape), list(a.shape), capi.BF16, dev)
    return CudaTensor.from_cpu(a, list(a.shape), capi.F32, dev)


def bf16(a):
    return bf16_to_f32(f32_to_bf16(np.asarray(a, np.float32))).reshape(np.shape(a))


def zeros(dev, *shape):
    from crabml_b200 import CudaTensor
    t = CudaTensor.alloc(list(shape), capi.F32, dev)
    seqops.tensor_zero(t)
    return t


def out(t, *shape):
    return t.export().reshape(shape)


# ---- elementwise, norms --------------------------------------------------------------------------------------------------------------
def test_activations_in_place(dev):
    z = np.linspace(-5, 5, 71)
    want = {capi.ACT_NONE: z, capi.ACT_SILU: R.silu(z), capi.ACT_SIGMOID: R.sigmoid(z), capi.ACT_RELU_SQUARED: R.relu_squared(z)}
    for act, w in want.items():
        assert np.abs(seqops.activate_inplace(T32(dev, z), act).export() - w).max() < 1e-5, act


def test_softcap(dev):
    z = np.array([0.0, 0.3, -4.0, 29.0, 500.0, -1e4])
    assert np.abs(seqops.softcap_inplace(T32(dev, z), 7.5).export() - R.soft_cap(z, 7.5)).max() < 1e-5
    with pytest.raises(capi.TensorError):
        seqops.softcap_inplace(T32(dev, z), 0.0)


@pytest.mark.parametrize("rows,cols", [(1, 5), (7, 511), (3, 512), (1, 1000), (40, 2048)])
def test_normed_output_joins_the_residual(dev, rows, cols):
    rng = np.random.default_rng(cols)
    x, y, w = rng.standard_normal((rows, cols)), rng.standard_normal((rows, cols)) * 4, rng.standard_normal(cols)
    got = out(seqops.rms_norm_gain(T32(dev, x), T32(dev, y), T32(dev, w), 1e-3, accumulate=True), rows, cols)
    assert np.abs(got - (x + R.rms_norm(y, w, 1e-3))).max() < 1e-5
    assert np.abs(out(seqops.group_rms_norm(T32(dev, y), T32(dev, w), 1, 1e-3), rows, cols) - R.rms_norm(y, w, 1e-3)).max() < 1e-5


@pytest.mark.parametrize("rows,cols,groups,wider", [(5, 24, 3, 7), (2, 1024, 2, 0), (9, 600, 1, 33), (1, 8, 8, 4)])
def test_gate_then_norm_reads_its_gate_from_a_wider_matrix(dev, rows, cols, groups, wider):
    from crabml_b200 import TensorStrider
    rng = np.random.default_rng(cols + wider)
    y, w = rng.standard_normal((rows, cols)), rng.standard_normal(cols)
    src = rng.standard_normal((rows, cols + wider))
    gate = T32(dev, src).with_strider(TensorStrider([rows, cols], [cols + wider, 1]))
    got = out(seqops.gated_group_rms_norm(T32(dev, y), gate, T32(dev, w), groups, 1e-4), rows, cols)
    assert np.abs(got - R.gate_then_group_norm(y, src[:, :cols], w, groups, 1e-4)).max() < 2e-5


# ---- convolution -----------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("K", [1, 2, 4, 6])
@pytest.mark.parametrize("portions", [[30], [1] * 30, [8, 9, 2, 1, 10], [2] * 15, [3, 4, 5, 6, 7, 5]])
def test_convolution_over_a_column_block_in_portions(dev, K, portions):
    rng = np.random.default_rng(K)
    C, col0, tail_cols, T = 11, 5, 3, 30
    src, w, b = rng.standard_normal((T, col0 + C + tail_cols)), rng.standard_normal((C, K)), rng.standard_normal(C)
    tail = zeros(dev, K - 1, C) if K > 1 else None
    got, at = [], 0
    for n in portions:
        got.append(out(seqops.short_conv_cols(T32(dev, src[at:at + n]), col0, T32(dev, w), T32(dev, b), tail), n, C))
        at += n
    x = src[:, col0:col0 + C]
    assert np.abs(np.concatenate(got) - R.silu(R.causal_conv(x, w, b))).max() < 1e-5
    if K > 1:
        assert np.allclose(out(tail, K - 1, C), x[T - K + 1:].astype(np.float32))
    with pytest.raises(capi.TensorError):
        seqops.short_conv_cols(T32(dev, src), col0 + tail_cols + 1, T32(dev, w), T32(dev, b), tail)


# ---- state space --------------------------------------------------------------------------------------------------------------------------
def scan_inputs(rng, T, H, P, N, G):
    return rng.standard_normal((T, H, P)), rng.standard_normal((T, G, N)) / np.sqrt(N), rng.standard_normal((T, G, N)), rng.standard_normal((T, H)), rng.uniform(-2, 1, H), rng.uniform(-3, 0, H), rng.standard_normal(H)


@pytest.mark.parametrize("H,P,N,G", [(4, 6, 10, 2), (1, 1, 1, 1), (6, 33, 48, 3), (4, 64, 128, 1), (2, 70, 64, 2), (3, 40, 32, 1), (8, 16, 130, 4)])
def test_scan_with_steps_from_a_column_block_in_portions(dev, H, P, N, G):
    rng = np.random.default_rng(H * P + N)
    T, extra = 45, 9
    x, B, C, dt, a_log, bias, d = scan_inputs(rng, T, H, P, N, G)
    want = R.state_space(x, B, C, R.softplus(dt + bias), a_log, d).reshape(T, -1)
    xbc = np.concatenate([x.reshape(T, -1), B.reshape(T, -1), C.reshape(T, -1)], 1)
    src = np.concatenate([rng.standard_normal((T, extra)), dt], 1)
    first = None
    for portions in ([T], [1] * T, [16, 17, 2, 10], [2] * 22 + [1], [30] + [1] * 15):
        S, got, at = zeros(dev, H, N, P), [], 0
        for n in portions:
            got.append(out(seqops.state_space_scan_cols(T32(dev, xbc[at:at + n]), T32(dev, src[at:at + n]), extra, T32(dev, bias), T32(dev, a_log), T32(dev, d), S, H, G, N, P), n, H * P))
            at += n
        got = np.concatenate(got)
        assert np.abs(got - want).max() < 2e-5 * max(1.0, np.abs(want).max()), portions
        first = got if first is None else first
        assert np.array_equal(got, first)                              # one order of operations per token: the same bits however it is cut


def test_scan_remembers_a_far_token_and_forgets_by_its_decay(dev):
    """one head; an outer product of weight 1 at token 0, nothing afterwards, read out 600 tokens later in a prompt and token by token"""
    T, N, P = 601, 4, 3
    rate = np.log(1e-3)                                                # decay per token exp(-1e-3 d)
    dt = np.full((T, 1), 50.0); dt[1:] = 0.5                           # softplus(50) = 50, softplus(0.5) = 0.974
    x, B, C = np.zeros((T, 1, P)), np.zeros((T, 1, N)), np.zeros((T, 1, N))
    x[0, 0], B[0, 0, 1], C[:, 0, 1] = [1.0, -2.0, 3.0], 1.0, 1.0
    z = np.zeros(1)
    want = R.state_space(x, B, C, R.softplus(dt), np.array([rate]), z).reshape(T, P)
    xbc = np.concatenate([x.reshape(T, -1), B.reshape(T, -1), C.reshape(T, -1)], 1)
    assert np.abs(want[600]).min() > 10
    for portions in ([T], [500] + [1] * 101):
        S, got, at = zeros(dev, 1, N, P), [], 0
        for n in portions:
            got.append(out(seqops.state_space_scan_cols(T32(dev, xbc[at:at + n]), T32(dev, dt[at:at + n]), 0, T32(dev, z), T32(dev, [rate]), None, S, 1, 1, N, P), n, P)); at += n
        assert np.abs(np.concatenate(got) - want).max() < 2e-3         # of values around 100: 600 products of decays


# ---- latent attention ------------------------------------------------------------------------------------------------------------------------
class Mixer:
    """the op chain of one latent-attention layer on one sequence, fed in portions (what the runner's mixer does); `shared`: another Mixer whose
    ring this layer reads"""

    def __init__(self, dev, w, m, ring_rows, eps=1e-5, expand_over=64, shared=None):
        from crabml_b200 import CudaTensor
        self.dev, self.m, self.eps, self.at, self.expand_over, self.rows, self.shared = dev, m, eps, 0, expand_over, ring_rows, shared
        own = ["m.dkv"] if shared is None else []
        self.stack = T32(dev, np.concatenate([w[n] for n in ["m.q", "m.g"] + own]))
        self.w = {k: T32(dev, v) for k, v in w.items()}
        uk = np.asarray(w["m.uk"], np.float32).reshape(m["heads"], m["dim"], m["kv_rank"])
        self.w["m.uk_t"] = T32(dev, np.ascontiguousarray(uk.transpose(0, 2, 1)).reshape(-1, m["dim"]))
        f, self.mag = rotary.table_of(m["rot"]) if m["rot_dim"] else (None, 1.0)
        self.f = T32(dev, f) if m["rot_dim"] else None
        self.ring = CudaTensor.alloc([ring_rows, m["kv_rank"] + m["rot_dim"]], capi.F32, dev) if shared is None else shared.ring

    def feed(self, h):
        from crabml_b200 import TensorStrider
        m, w, n = self.m, self.w, h.shape[0]
        H, dn, dr, dv, kr = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        all_ = self.stack.matmul_vec(T32(self.dev, h))
        qc, gc = H * (dn + dr), H * dv
        if n * H > self.expand_over:              # many rows: per-head keys and values of the ring's rows, then attention per head
            parts = seqops.split_cols(all_, [qc, gc] + ([kr + dr] if self.shared is None else []))
            if self.shared is None:
                seqops.latent_ring_append(self.ring, parts[2], w["m.dkv.norm"], self.eps, kr, self.f, self.mag, self.at)
            q = seqops.rope_pairs(parts[0], H, dn + dr, dn, self.f, self.mag, self.at) if self.f is not None else parts[0]
            rows = min(self.rows, self.at + n)
            lat = self.ring.with_strider(TensorStrider([rows, kr], [kr + dr, 1])).contiguous()
            keys = seqops.head_concat_shared(w["m.uk"].matmul_vec(lat), self.ring, H, kr, dr)
            o = seqops.window_attention_sink(q, keys, w["m.uv"].matmul_vec(lat), self.at, H, H, dn + dr, dv, 0, m["scale"], sink=w["m.sink"])
            o = seqops.gated_sum(o, o, g1=parts[1], accumulate=False)
        else:                                     # few rows: fold + cache write in one kernel, the gate in the last product
            kv = all_ if self.shared is None else None
            ql = seqops.latent_query_append(all_, 0, w["m.uk_t"], H, dr, self.f, self.mag, self.at, kv, qc + gc, self.ring, w.get("m.dkv.norm"), self.eps)
            ol = seqops.window_attention_sink(ql, self.ring, None, self.at, H, 1, kr + dr, kr, 0, m["scale"], sink=w["m.sink"])
            o = seqops.head_project_gated(ol, w["m.uv"], H, all_, qc)
        res = w["m.o"].matmul_vec(o).export().reshape(n, -1)
        self.at += n
        return res


def attention_weights(rng, D, m, own=True):
    def mat(o, i):
        return bf16(rng.standard_normal((o, i)) / np.sqrt(i))
    H, dn, dr, dv, kr = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    w = {"m.q": mat(H * (dn + dr), D), "m.g": mat(H * dv, D), "m.uk": mat(H * dn, kr), "m.uv": mat(H * dv, kr), "m.o": mat(D, H * dv), "m.sink": rng.standard_normal(H) * 2}
    if own:
        w.update({"m.dkv": mat(kr + dr, D), "m.dkv.norm": 1 + 0.2 * rng.standard_normal(kr)})
    return w


def sizes(H, dn, dr, dv, kr, base=300.0):
    return {"heads": H, "dim": dn, "rot_dim": dr, "vdim": dv, "kv_rank": kr, "scale": 1.0 / np.sqrt(dn + dr), "rot": {"dims": dr, "base": base}}


def feed_all(mx, h, portions):
    return np.concatenate([mx.feed(h[a:a + n]) for a, n in zip(np.cumsum([0] + portions[:-1]), portions)])


PORTIONS = [[61], [1] * 61, [29] + [1] * 32, [2, 3, 30, 2, 17, 1, 1, 5], [2] * 30 + [1]]


@pytest.mark.parametrize("H,dn,dr,dv,kr", [(3, 8, 4, 10, 20), (1, 16, 2, 5, 9), (8, 24, 12, 40, 80), (64, 2, 2, 2, 6), (16, 4, 4, 40, 36), (5, 7, 6, 3, 11), (2, 4, 0, 6, 8)])
def test_latent_attention_and_a_layer_that_shares_its_cache(dev, H, dn, dr, dv, kr):
    rng = np.random.default_rng(H * 7 + kr)
    D, T = 24, 61
    m, m2 = sizes(H, dn, dr, dv, kr), sizes(H % 4 + 1, dn + 3, dr, dv + 1, kr)
    w, w2 = attention_weights(rng, D, m), attention_weights(rng, D, m2, own=False)
    h, h2 = rng.standard_normal((T, D)).astype(np.float32).astype(np.float64), rng.standard_normal((T, D)).astype(np.float32).astype(np.float64)
    lat = R.latent_rows(h, w, "m.", m, 1e-5)
    want, want2 = R.latent_attention(h, lat, w, "m.", m), R.latent_attention(h2, lat, w2, "m.", m2)
    for expand_over in (64, 0, 10 ** 9):              # the runner's rule, every pass expanded, every pass folded
        for portions in PORTIONS:
            mx = Mixer(dev, w, m, T, expand_over=expand_over)
            sh = Mixer(dev, w2, m2, T, expand_over=expand_over, shared=mx)
            got, got2 = [], []
            for a, n in zip(np.cumsum([0] + portions[:-1]), portions):         # the layers of one pass run one after the other
                got.append(mx.feed(h[a:a + n])); got2.append(sh.feed(h2[a:a + n]))
            assert np.abs(np.concatenate(got) - want).max() < 3e-5 * max(1.0, np.abs(want).max()), (expand_over, portions)
            assert np.abs(np.concatenate(got2) - want2).max() < 3e-5 * max(1.0, np.abs(want2).max()), (expand_over, portions)


def _towering_key(dev, T, j_star, portions, sink=-1e30, expand_over=8):
    """One head.  Every query scores 0 with every key but the one at j_star, which it scores with 60: whoever sees j_star returns its value."""
    m = {"heads": 1, "dim": 2, "rot_dim": 2, "vdim": 2, "kv_rank": 2, "scale": 1.0, "rot": {"dims": 2, "base": 10.0}}
    D = 4
    w = {"m.q": np.zeros((4, D)), "m.g": np.zeros((2, D)), "m.dkv": np.eye(4, D), "m.dkv.norm": np.ones(2), "m.uk": np.zeros((2, 2)), "m.uv": np.eye(2), "m.sink": np.array([sink]),
         "m.o": np.eye(D, 2)}
    w["m.q"][0, 3] = 60.0 / np.sqrt(2.0)                       # a query reads the constant fourth column
    w["m.uk"][0, 1] = 1.0                                      # a key is its latent's second coordinate
    w["m.dkv"][3] = 0.0                                        # no rotated part: the fourth column does not reach the cache
    h = np.zeros((T, D)); h[:, 0] = 1.0; h[:, 3] = 1.0
    h[j_star, :2] = (0.0, 1.0)
    got = feed_all(Mixer(dev, w, m, T, expand_over=expand_over), h, portions)
    lat = R.latent_rows(h, w, "m.", m, 1e-5)
    assert np.abs(got - R.latent_attention(h, lat, w, "m.", m)).max() < 1e-4
    return got[:, :2]


@pytest.mark.parametrize("portions", [[700], [640] + [1] * 60, [256, 256, 188], [63, 1, 64, 1, 2, 569], [2] * 350])
@pytest.mark.parametrize("j_star", [0, 1, 63, 64, 257])
def test_a_key_far_away_is_seen_from_its_own_position_on_and_never_before(dev, portions, j_star):
    o = _towering_key(dev, 700, j_star, portions)
    v = np.sqrt(2.0) / 2                                       # the normed latent (0, sqrt 2), gated by 1/2
    assert np.abs(o[:j_star, 1]).max(initial=0.0) < 1e-6       # nobody before it
    assert (np.abs(o[j_star:, 1] - v) < 1e-3).all() and np.abs(o[j_star:, 0]).max() < 1e-3


def test_sink_takes_its_share_of_many_keys_and_a_tower_beats_it(dev):
    T = 130
    for portions in ([T], [100] + [1] * 30):
        o = _towering_key(dev, T, 40, portions, sink=np.log(25.0))
        v = np.sqrt(2.0) / 2
        for i in (0, 5, 39):                                   # i + 1 keys of score 0 beside a sink of 25
            assert abs(o[i, 0] - v * (i + 1) / (i + 1 + 25.0)) < 1e-4
        assert abs(o[T - 1, 1] - v) < 1e-3
        o = _towering_key(dev, T, 40, portions, sink=80.0)     # higher than the tower: next to nothing is left
        assert np.abs(o).max() < 1e-6


def test_rotated_part_alone_finds_a_key_by_its_distance(dev):
    """queries and keys agree only in the rotated pair: the score is 1000 cos(i - j), largest at i = j, whatever the position; 44 tokens back (seven
    full turns) it is nearly as large again"""
    m = {"heads": 1, "dim": 1, "rot_dim": 2, "vdim": 1, "kv_rank": 1, "scale": 1000.0, "rot": {"dims": 2, "base": 10.0}}
    D, T = 3, 150
    w = {"m.q": np.zeros((3, D)), "m.g": np.zeros((1, D)), "m.dkv": np.zeros((3, D)), "m.dkv.norm": np.ones(1), "m.uk": np.zeros((1, 1)), "m.uv": np.ones((1, 1)), "m.sink": np.array([-1e30]),
         "m.o": np.eye(D, 1)}
    w["m.q"][1, 0] = w["m.dkv"][1, 0] = 1.0
    w["m.dkv"][0, 1] = 1.0
    h = np.zeros((T, D)); h[:, 0] = 1.0; h[:, 1] = np.where(np.arange(T) % 2, 1.0, -1.0)
    want = R.latent_attention(h, R.latent_rows(h, w, "m.", m, 1e-5), w, "m.", m)
    assert np.abs(want[:44, 0] - h[:44, 1] / 2).max() < 1e-3           # until then every position returns its own value
    for portions in ([T], [100] + [1] * 50, [64, 1, 1, 84]):
        got = feed_all(Mixer(dev, w, m, T, expand_over=8), h, portions)
        assert np.abs(got - want).max() < 5e-3                         # scores of 1000 times a 32-bit cosine


def test_latent_ops_refuse_what_does_not_fit(dev):
    rng = np.random.default_rng(0)
    src, ukt, ring, f = T32(dev, rng.standard_normal((3, 20))), T32(dev, rng.standard_normal((2 * 4, 3))), zeros(dev, 8, 6), T32(dev, [1.0])
    ok = seqops.latent_query_append(src, 2, ukt, 2, 2, f, 1.0, 0, src, 14, ring, None, 1e-5)
    assert ok.shape() == [3, 12]
    for bad in (dict(q_col0=11), dict(kv_col0=15), dict(ring=zeros(dev, 8, 7)), dict(ring=zeros(dev, 2, 6)), dict(norm_w=T32(dev, np.ones(3))), dict(freq=T32(dev, [1.0, 1.0]))):
        kw = dict(q_src=src, q_col0=2, uk_t=ukt, n_heads=2, rest=2, freq=f, mag=1.0, pos0=0, kv_src=src, kv_col0=14, ring=ring, norm_w=None, eps=1e-5)
        kw.update(bad)
        with pytest.raises(capi.TensorError):
            seqops.latent_query_append(**kw)
    with pytest.raises(capi.TensorError):
        seqops.head_project_gated(T32(dev, rng.standard_normal((3, 8))), T32(dev, rng.standard_normal((10, 4))), 2, src, 11)


# ---- feed-forwards ------------------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("E,top,n_shared,D", [(6, 2, 2, 24), (16, 1, 0, 36), (5, 5, 3, 13), (1, 1, 1, 7), (40, 7, 40, 64), (128, 8, 1, 512)])
@pytest.mark.parametrize("T", [1, 3, 130])
def test_router_with_shared_slots(dev, E, top, n_shared, D, T):
    rng = np.random.default_rng(E + T)
    x, wr, sg = (rng.standard_normal(s).astype(np.float32) for s in ((T, D), (E, D), (D,)))
    ids, wts = seqops.moe_route_shared(T32(dev, x), T32(dev, wr), None, top, shared_gate=T32(dev, sg) if n_shared else None, n_shared=n_shared, renormalise=True, renorm_eps=1e-20,
                                       scale=1.7)
    ids, wts = ids.export().view(np.int32).reshape(T, -1), out(wts, T, -1)
    rid, rw = R.route(x.astype(np.float64), wr.astype(np.float64), top, 1.7)
    assert np.array_equal(ids[:, :top], rid) and np.abs(wts[:, :top] - rw).max() < 2e-5
    assert np.array_equal(ids[:, top:], np.tile(E + np.arange(n_shared), (T, 1)))
    assert np.abs(wts[:, top:] - R.sigmoid(x.astype(np.float64) @ sg.astype(np.float64))[:, None]).max(initial=0.0) < 2e-5
    # a token's choice does not depend on the pass it comes with
    i1, w1 = seqops.moe_route_shared(T32(dev, x[-1:]), T32(dev, wr), None, top, shared_gate=T32(dev, sg) if n_shared else None, n_shared=n_shared, renormalise=True, renorm_eps=1e-20,
                                     scale=1.7)
    assert np.array_equal(i1.export().view(np.int32), ids[-1]) and np.array_equal(w1.export(), wts[-1])


def test_shared_slots_without_a_gate_weigh_one_and_scale_zero_counts_as_one(dev):
    rng = np.random.default_rng(1)
    x, wr = rng.standard_normal((4, 12)), rng.standard_normal((3, 12))
    _, wts = seqops.moe_route_shared(T32(dev, x), T32(dev, wr), None, 2, n_shared=2, renormalise=True, scale=0.0)
    assert np.allclose(out(wts, 4, 4)[:, 2:], 1.0) and np.allclose(out(wts, 4, 4)[:, :2].sum(1), 1.0, atol=1e-6)
    with pytest.raises(capi.TensorError):
        seqops.moe_route_shared(T32(dev, x), T32(dev, wr), None, 2, shared_gate=T32(dev, np.ones(12)), n_shared=0)


@pytest.mark.parametrize("dtype", [capi.F32, capi.BF16])
@pytest.mark.parametrize("T,D,E,ff,slots", [(1, 24, 4, 10, 3), (3, 13, 5, 7, 2), (1, 256, 6, 264, 6), (2, 512, 3, 64, 3), (200, 64, 5, 64, 3), (130, 128, 4, 192, 1), (90, 72, 3, 56, 2)])
def test_experts_of_plain_units(dev, dtype, T, D, E, ff, slots):
    from crabml_b200 import CudaTensor
    rng = np.random.default_rng(T + D)
    x = rng.standard_normal((T, D)) * 1.5
    wu, wd = bf16(rng.standard_normal((E, ff, D)) / np.sqrt(D)), bf16(rng.standard_normal((E, D, ff)) / np.sqrt(ff))
    ids = np.stack([rng.permutation(max(E, slots))[:slots] % E for _ in range(T)]).astype(np.int32)
    wts = rng.uniform(0.1, 1.0, (T, slots))
    got = out(seqops.moe_experts_act(T32(dev, x), CudaTensor.from_cpu(ids, [T, slots], capi.I32, dev), T32(dev, wts), W(dev, wu.reshape(E * ff, D), dtype), W(dev, wd.reshape(E * D, ff), dtype),
                                     E, ff, capi.ACT_RELU_SQUARED), T, D)
    xin = (bf16(x) if dtype == capi.BF16 else x.astype(np.float32)).astype(np.float64)
    want = np.zeros((T, D))
    for t in range(T):
        for e, a in zip(ids[t], wts[t].astype(np.float32)):
            hid = R.relu_squared(wu[e].astype(np.float64) @ xin[t])
            want[t] += a * (wd[e].astype(np.float64) @ (bf16(hid) if dtype == capi.BF16 else hid))
    tol = 2e-3 if dtype == capi.BF16 else 3e-5                # a hidden unit next to a bfloat16 rounding boundary may fall on the other side
    assert np.abs(got - want).max() < tol * max(1.0, np.abs(want).max())


@pytest.mark.parametrize("dtype", [capi.F32, capi.BF16])
@pytest.mark.parametrize("T", [1, 7, 8, 31, 32, 200])
@pytest.mark.parametrize("D,ff", [(64, 128), (36, 40), (13, 9), (128, 72)])
def test_dense_feed_forward_of_plain_units(dev, dtype, T, D, ff):
    rng = np.random.default_rng(T + D)
    x = rng.standard_normal((T, D))
    wu, wd = bf16(rng.standard_normal((ff, D)) / np.sqrt(D)), bf16(rng.standard_normal((D, ff)) / np.sqrt(ff))
    got = out(seqops.feed_forward_act(T32(dev, x), W(dev, wu, dtype), W(dev, wd, dtype), capi.ACT_RELU_SQUARED), T, D)
    xin = (bf16(x) if dtype == capi.BF16 else x.astype(np.float32)).astype(np.float64)
    hid = R.relu_squared(xin @ wu.T.astype(np.float64))
    want = (bf16(hid) if dtype == capi.BF16 else hid) @ wd.T.astype(np.float64)
    assert np.abs(got - want).max() < (2e-3 if dtype == capi.BF16 else 3e-5) * max(1.0, np.abs(want).max())
    # a row's result does not depend on the rows it comes with, beyond rounding
    one = out(seqops.feed_forward_act(T32(dev, x[-1:]), W(dev, wu, dtype), W(dev, wd, dtype), capi.ACT_RELU_SQUARED), 1, D)
    assert np.abs(one[0] - got[-1]).max() < (2e-3 if dtype == capi.BF16 else 3e-5) * max(1.0, np.abs(want).max())
