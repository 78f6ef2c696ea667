"""The mechanisms the Vadodra family added to include/crabml_seqops.h or uses in another form, each alone, against its function in the plain
reference (tests/vadodra_ref.py).  Where random inputs would hide a fault (a far key, a window's edge, a clamped unit) the inputs are made so that
it shows."""
import numpy as np
import pytest

from crabml_b200 import capi, rotary, seqops
from crabml_b200.safetensors import bf16_to_f32, f32_to_bf16
from tests import vadodra_ref as R
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
    return bf16_to_f32(f32_to_bf16(np.asarray(a, np.float32))).reshape(np.shape(a)).astype(np.float64)


def zeros(dev, *shape):
    from crabml_b200 import CudaTensor
    t = CudaTensor.alloc(list(shape), capi.F32, dev)
    seqops.tensor_zero(t)
    return t


def out(t, *shape):
    return t.export().reshape(shape)


def f32(a):
    return np.asarray(a, np.float32).astype(np.float64)


# ---- the products around a layer ----------------------------------------------------------------------------------------------------------
ROWS = [1, 3, 7, 8, 31, 32, 130, 200]


@pytest.mark.parametrize("dtype", [capi.F32, capi.BF16])
@pytest.mark.parametrize("k,m", [(64, 128), (36, 40), (13, 9), (1, 1), (128, 600), (520, 77), (9000, 5), (256, 5000)])
def test_norm_and_product(dev, dtype, k, m):
    rng = np.random.default_rng(k + m)
    w = bf16(rng.standard_normal((m, k)) / np.sqrt(k))
    g, b = f32(1 + 0.3 * rng.standard_normal(k)), f32(rng.standard_normal(k))
    wd = W(dev, w, dtype)
    x = f32(rng.standard_normal((200, k)) * 3 + 50.0)                # a mean far from 0
    for bias in (None, b):
        h = R.layer_norm(x, g, 1e-5) + (0 if bias is None else bias)
        want = (bf16(h) if dtype == capi.BF16 else h) @ w.T
        tol = (4e-3 if dtype == capi.BF16 else 1e-4) * max(1.0, np.abs(want).max())      # an operand next to a rounding boundary may fall on the other side
        for T in ROWS if k < 9000 else [1, 8]:
            got = out(seqops.layer_norm_product(T32(dev, x[:T]), T32(dev, g), None if bias is None else T32(dev, bias), 1e-5, wd), T, m)
            assert np.abs(got - want[:T]).max() < tol, (T, np.abs(got - want[:T]).max())


@pytest.mark.parametrize("dtype", [capi.F32, capi.BF16])
@pytest.mark.parametrize("ca,ff,m", [(64, 128, 64), (33, 17, 36), (10, 0, 24), (64, 0, 130), (1, 1, 1), (96, 160, 700), (40, 24, 5000), (9000, 21000, 3)])
def test_joined_product_with_gated_units(dev, dtype, ca, ff, m):
    rng = np.random.default_rng(ca + ff + m)
    w = bf16(rng.standard_normal((m, ca + ff)) / np.sqrt(ca + ff))
    wd = W(dev, w, dtype)
    rows = [1, 2, 9] if ca == 9000 else ROWS
    N = max(rows)
    a, x0 = f32(rng.standard_normal((N, ca))), f32(rng.standard_normal((N, m)))
    src = f32(rng.standard_normal((N, 2 * ff + 11)) * 2)               # units well beyond the limit on both sides
    gc, uc = (3, ff + 5)
    for limit in (0.9, 30.0):
        unit = R.clamped_unit(src[:, gc:gc + ff], src[:, uc:uc + ff], limit)
        op = np.concatenate([a, unit], 1)
        want = x0 + (bf16(op) if dtype == capi.BF16 else op) @ w.T
        tol = (4e-3 if dtype == capi.BF16 else 5e-5) * max(1.0, np.abs(want).max())
        for T in rows:
            x = T32(dev, x0[:T])
            kw = dict(src=T32(dev, src[:T]), gate_col0=gc, up_col0=uc, ff=ff, act=capi.ACT_SWISH, alpha=1.702, limit=limit, up_shift=1.0) if ff else {}
            got = out(seqops.joined_product_accumulate(x, wd, T32(dev, a[:T]), **kw), T, m)
            assert np.abs(got - want[:T]).max() < tol, (T, limit, np.abs(got - want[:T]).max())


def test_joined_product_takes_other_units(dev):
    rng = np.random.default_rng(3)
    a, src, w = f32(rng.standard_normal((4, 6))), f32(rng.standard_normal((4, 10))), f32(rng.standard_normal((7, 11)))
    got = out(seqops.joined_product_accumulate(zeros(dev, 4, 7), T32(dev, w), T32(dev, a), T32(dev, src), 0, 5, 5, capi.ACT_GELU_TANH), 4, 7)
    z = src[:, :5]
    unit = 0.5 * z * (1 + np.tanh(np.sqrt(2 / np.pi) * (z + 0.044715 * z ** 3))) * src[:, 5:]
    assert np.abs(got - np.concatenate([a, unit], 1) @ w.T).max() < 1e-5


def test_a_row_gives_the_same_bits_in_every_call_of_few_rows(dev):
    rng = np.random.default_rng(5)
    x, g, w = f32(rng.standard_normal((7, 300))), f32(rng.standard_normal(300)), bf16(rng.standard_normal((90, 300)))
    for dtype in (capi.F32, capi.BF16):
        wd = W(dev, w, dtype)
        whole = out(seqops.layer_norm_product(T32(dev, x), T32(dev, g), None, 1e-5, wd), 7, 90)
        for t in range(7):
            assert np.array_equal(out(seqops.layer_norm_product(T32(dev, x[t:t + 1]), T32(dev, g), None, 1e-5, wd), 1, 90)[0], whole[t])


def test_products_refuse_what_does_not_fit(dev):
    x, g, w = zeros(dev, 3, 8), zeros(dev, 8), zeros(dev, 5, 8)
    for bad in ((zeros(dev, 3, 7), g, None, w), (x, zeros(dev, 7), None, w), (x, g, zeros(dev, 9), w)):
        with pytest.raises(capi.TensorError):
            seqops.layer_norm_product(bad[0], bad[1], bad[2], 1e-5, bad[3])
    dst, a, src = zeros(dev, 3, 5), zeros(dev, 3, 6), zeros(dev, 3, 9)
    for kw in (dict(gate_col0=0, up_col0=8, ff=2), dict(gate_col0=-1, up_col0=0, ff=2), dict(gate_col0=0, up_col0=0, ff=3), dict(src=zeros(dev, 2, 9), gate_col0=0, up_col0=2, ff=2)):
        kw = dict({"src": src}, **kw)
        with pytest.raises(capi.TensorError):
            seqops.joined_product_accumulate(dst, w, a, **kw)


# ---- column blocks ----------------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("pairing", [capi.ROPE_NEIGHBOURS, capi.ROPE_HALVES])
@pytest.mark.parametrize("norm", [capi.QK_NORM_NONE, capi.QK_NORM_HEAD, capi.QK_NORM_ROW])
def test_prepared_columns_are_the_prepared_tensors(dev, norm, pairing):
    rng = np.random.default_rng(norm)
    T, H, G, dk, dv, ring, pos0 = 5, 6, 2, 10, 7, 9, 7
    q, k, v = (rng.standard_normal((T, n)) for n in (H * dk, G * dk, G * dv))
    qw, kw = (rng.standard_normal(n) for n in ((H * dk, G * dk) if norm == capi.QK_NORM_ROW else (dk, dk)))
    args = dict(qk_norm=norm, eps=1e-4, freq=T32(dev, [1.0, 0.3]), pairing=pairing, offset=3, mag=1.2)
    if norm != capi.QK_NORM_NONE:
        args.update(q_w=T32(dev, qw), k_w=T32(dev, kw))
    kr, vr, kr2, vr2 = zeros(dev, ring, G * dk), zeros(dev, ring, G * dv), zeros(dev, ring, G * dk), zeros(dev, ring, G * dv)
    want = out(seqops.qk_prepare_append(T32(dev, q), T32(dev, k), T32(dev, v), kr, vr, pos0, H, G, dk, dv, **args), T, -1)
    src = T32(dev, np.concatenate([rng.standard_normal((T, 3)), v, q, rng.standard_normal((T, 2)), k], 1))
    got = out(seqops.qk_prepare_append_cols(src, 3 + G * dv, 5 + G * dv + H * dk, 3, kr2, vr2, pos0, H, G, dk, dv, **args), T, -1)
    assert np.array_equal(got, want) and np.array_equal(kr.export(), kr2.export()) and np.array_equal(vr.export(), vr2.export())
    with pytest.raises(capi.TensorError):
        seqops.qk_prepare_append_cols(src, 3 + G * dv, 6 + G * dv + H * dk, 3, kr2, vr2, pos0, H, G, dk, dv, **args)


def test_head_gate_from_columns(dev):
    rng = np.random.default_rng(2)
    x, g = rng.standard_normal((5, 12)), rng.standard_normal((5, 10))
    got = out(seqops.head_gate_cols(T32(dev, x), T32(dev, g), 4, 3), 5, 3, 4)
    assert np.abs(got - x.reshape(5, 3, 4) * R.sigmoid(g[:, 4:7])[..., None]).max() < 1e-6
    with pytest.raises(capi.TensorError):
        seqops.head_gate_cols(T32(dev, x), T32(dev, g), 8, 3)


@pytest.mark.parametrize("T", [1, 3, 20])
def test_head_product_gated_by_one_number_per_head(dev, T):
    rng = np.random.default_rng(T)
    H, n_in, n_out = 5, 9, 6
    x, w, g = rng.standard_normal((T, H * n_in)), rng.standard_normal((H * n_out, n_in)), rng.standard_normal((T, 8))
    want = np.einsum("thi,hoi->tho", x.reshape(T, H, n_in), w.reshape(H, n_out, n_in)) * R.sigmoid(g[:, 2:7])[..., None]
    assert np.abs(out(seqops.head_project_head_gated(T32(dev, x), T32(dev, w), H, T32(dev, g), 2), T, H, n_out) - want).max() < 2e-5
    with pytest.raises(capi.TensorError):
        seqops.head_project_head_gated(T32(dev, x), T32(dev, w), H, T32(dev, g), 4)


# ---- window attention over raw keys as values ---------------------------------------------------------------------------------------------------
class WindowMixer:
    """the op chain of one window-attention layer on one sequence, fed in portions"""

    def __init__(self, dev, w, m, chunk, eps=1e-5):
        self.dev, self.m, self.eps, self.at = dev, m, eps, 0
        self.stack = T32(dev, np.concatenate([w["m.q"], w["m.k"]]))
        self.w = {k: T32(dev, v) for k, v in w.items()}
        f, self.mag = rotary.table_of(m["rot"])
        self.f = T32(dev, f)
        ring = m["mask"]["size"] - 1 + chunk
        self.kr, self.vr = zeros(dev, ring, m["kv_heads"] * m["dim"]), zeros(dev, ring, m["kv_heads"] * m["dim"])

    def feed(self, h):
        m, n = self.m, h.shape[0]
        H, G, d = m["heads"], m["kv_heads"], m["dim"]
        src = self.stack.matmul_vec(T32(self.dev, h))
        q = seqops.qk_prepare_append_cols(src, 0, H * d, H * d, self.kr, self.vr, self.at, H, G, d, d, capi.QK_NORM_HEAD, self.w["m.q.norm"], self.w["m.k.norm"], self.eps, self.f,
                                          capi.ROPE_NEIGHBOURS, 0, self.mag)
        o = seqops.masked_attention_capped(q, self.kr, self.vr, self.at, H, G, d, d, m["scale"], window=m["mask"]["size"])
        self.at += n
        return self.w["m.o"].matmul_vec(o).export().reshape(n, -1)


def feed_all(mx, h, portions):
    return np.concatenate([mx.feed(h[a:a + n]) for a, n in zip(np.cumsum([0] + portions[:-1]), portions)])


PORTIONS = [[61], [1] * 61, [29] + [1] * 32, [2, 3, 30, 2, 17, 1, 1, 5], [2] * 30 + [1]]


@pytest.mark.parametrize("H,G,d,rot,size", [(6, 3, 10, 4, 7), (1, 1, 2, 2, 1), (8, 2, 16, 16, 16), (5, 5, 7, 6, 40), (16, 1, 32, 8, 64), (9, 3, 6, 2, 100), (64, 1, 4, 2, 5)])
def test_window_attention_layer(dev, H, G, d, rot, size):
    rng = np.random.default_rng(H + size)
    D, T = 20, 61
    m = {"heads": H, "kv_heads": G, "dim": d, "scale": 0.7 / np.sqrt(d), "mask": {"size": size}, "rot": {"dims": rot, "base": 300.0, "scaling": {"factor": 1.7}}}
    w = {n: f32(rng.standard_normal(s) / np.sqrt(s[-1])) for n, s in (("m.q", (H * d, D)), ("m.k", (G * d, D)), ("m.o", (D, H * d)))}
    w.update({"m.q.norm": f32(1 + 0.4 * rng.standard_normal(d)), "m.k.norm": f32(1 + 0.4 * rng.standard_normal(d))})
    h = f32(rng.standard_normal((T, D)))
    want = R.attention(h, w, "m.", m, 1e-5)
    for portions in PORTIONS:
        got = feed_all(WindowMixer(dev, w, m, max(portions)), h, portions)
        assert np.abs(got - want).max() < 5e-5 * max(1.0, np.abs(want).max()), portions


@pytest.mark.parametrize("size", [1, 2, 31, 32, 33, 64, 100])
@pytest.mark.parametrize("portions", [[300], [200] + [1] * 100, [64, 1, 63, 2, 170], [2] * 150])
def test_a_key_is_seen_to_the_last_row_of_its_window_and_not_beyond(dev, size, portions):
    """every query scores 0 with every key but the one at j_star, which it scores with about 60; the answer is then that key's raw row"""
    m = {"heads": 2, "kv_heads": 1, "dim": 4, "scale": 15.0, "mask": {"size": size}, "rot": {"dims": 2, "base": 10.0}}
    D, T = 4, 300
    w = {"m.q": np.zeros((8, D)), "m.k": np.zeros((4, D)), "m.q.norm": np.ones(4), "m.k.norm": np.ones(4), "m.o": np.eye(D, 8)}
    w["m.q"][3, 2] = w["m.q"][7, 2] = 1.0                              # a query is the unrotated fourth direction, read from the constant third column
    w["m.k"][2, 0] = w["m.k"][3, 1] = 1.0                              # a key is an unrotated direction as well: the third or, at j_star, the fourth
    for j_star in (0, 63, 64, 150):
        h = np.zeros((T, D)); h[:, 0] = 3.0; h[:, 2] = 1.0
        h[j_star, :2] = (0.0, 5.0)                                     # norms do not touch the values: 3 and 5 stay
        got = feed_all(WindowMixer(dev, w, m, max(portions)), h, portions)
        assert np.abs(got - R.attention(h, w, "m.", m, 1e-5)).max() < 1e-3
        seen = (np.arange(T) >= j_star) & (np.arange(T) < j_star + size)
        assert (np.abs(got[seen, 3] - 5.0) < 1e-2).all() and np.abs(got[~seen, 3]).max() < 1e-6 and (np.abs(got[~seen, 2] - 3.0) < 1e-5).all()


# ---- latent attention ------------------------------------------------------------------------------------------------------------------------
class LatentMixer:
    """the op chain of one latent-attention layer on one sequence, fed in portions; `shared`: another LatentMixer whose ring this layer reads"""

    def __init__(self, dev, w, m, ring_rows, eps=1e-5, expand_over=64, shared=None):
        from crabml_b200 import CudaTensor
        self.dev, self.m, self.eps, self.at, self.expand_over, self.rows, self.shared = dev, m, eps, 0, expand_over, ring_rows, shared
        self.stack = T32(dev, np.concatenate([w[n] for n in ["m.q", "m.g"] + (["m.dkv"] if shared is None else [])]))
        self.w = {k: T32(dev, v) for k, v in w.items()}
        uk = np.asarray(w["m.uk"], np.float32).reshape(m["heads"], m["dim"], m["kv_rank"])
        self.w["m.uk_t"] = T32(dev, np.ascontiguousarray(uk.transpose(0, 2, 1)).reshape(-1, m["dim"]))
        f, self.mag = rotary.table_of(m["rot"])
        self.f = T32(dev, f)
        self.ring = CudaTensor.alloc([ring_rows, m["kv_rank"] + m["rot_dim"]], capi.F32, dev) if shared is None else shared.ring

    def feed(self, h):
        from crabml_b200 import TensorStrider
        m, w, n = self.m, self.w, h.shape[0]
        H, dn, dr, dv, kr = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        src = self.stack.matmul_vec(T32(self.dev, h))
        qc, kv = H * (dn + dr), src if self.shared is None else None
        if n * H > self.expand_over:              # many rows: per-head keys and values of the ring's rows, then attention per head
            q = seqops.latent_prepare_append(src, 0, H, dn, dr, self.f, capi.ROPE_HALVES, self.mag, self.at, kv, qc + H, self.ring, w.get("m.dkv.norm"), self.eps)
            rows = min(self.rows, self.at + n)
            lat = self.ring.with_strider(TensorStrider([rows, kr], [kr + dr, 1])).contiguous()
            keys = seqops.head_concat_shared(w["m.uk"].matmul_vec(lat), self.ring, H, kr, dr)
            o = seqops.window_attention_sink(q, keys, w["m.uv"].matmul_vec(lat), self.at, H, H, dn + dr, dv, 0, m["scale"])
            o = seqops.head_gate_cols(o, src, qc, H)
        else:                                     # few rows: fold + cache write in one kernel, the gate in the last product
            ql = seqops.latent_query_append_paired(src, 0, w["m.uk_t"], H, dr, self.f, capi.ROPE_HALVES, self.mag, self.at, kv, qc + H, self.ring, w.get("m.dkv.norm"), self.eps)
            ol = seqops.window_attention_sink(ql, self.ring, None, self.at, H, 1, kr + dr, kr, 0, m["scale"])
            o = seqops.head_project_head_gated(ol, w["m.uv"], H, src, qc)
        self.at += n
        return w["m.o"].matmul_vec(o).export().reshape(n, -1)


def latent_weights(rng, D, m, own=True):
    def mat(o, i):
        return bf16(rng.standard_normal((o, i)) / np.sqrt(i))
    H, dn, dr, dv, kr = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    w = {"m.q": mat(H * (dn + dr), D), "m.g": mat(H, D), "m.uk": mat(H * dn, kr), "m.uv": mat(H * dv, kr), "m.o": mat(D, H * dv)}
    if own:
        w.update({"m.dkv": mat(kr + dr, D), "m.dkv.norm": f32(1 + 0.2 * rng.standard_normal(kr))})
    return w


def sizes(H, dn, dr, dv, kr, base=300.0):
    return {"heads": H, "dim": dn, "rot_dim": dr, "vdim": dv, "kv_rank": kr, "scale": 1.0 / np.sqrt(dn + dr), "rot": {"dims": dr, "base": base}}


@pytest.mark.parametrize("H,dn,dr,dv,kr", [(3, 8, 4, 10, 20), (1, 16, 2, 5, 9), (8, 24, 12, 40, 80), (64, 2, 2, 2, 6), (16, 4, 4, 40, 36), (5, 7, 6, 3, 11)])
def test_latent_attention_and_a_layer_that_shares_its_cache(dev, H, dn, dr, dv, kr):
    rng = np.random.default_rng(H * 7 + kr)
    D, T = 24, 61
    m, m2 = sizes(H, dn, dr, dv, kr), sizes(H % 4 + 1, dn + 3, dr, dv + 1, kr)
    w, w2 = latent_weights(rng, D, m), latent_weights(rng, D, m2, own=False)
    h, h2 = f32(rng.standard_normal((T, D))), f32(rng.standard_normal((T, D)))
    rows = R.latent_rows(h, w, "m.", m, 1e-5)
    want, want2 = R.latent_attention(h, rows, w, "m.", m), R.latent_attention(h2, rows, w2, "m.", m2)
    for expand_over in (64, 0, 10 ** 9):              # the runner's rule, every pass expanded, every pass folded
        for portions in PORTIONS:
            mx = LatentMixer(dev, w, m, T, expand_over=expand_over)
            sh = LatentMixer(dev, w2, m2, T, expand_over=expand_over, shared=mx)
            got, got2 = [], []
            for a, n in zip(np.cumsum([0] + portions[:-1]), portions):         # the layers of one pass run one after the other
                got.append(mx.feed(h[a:a + n])); got2.append(sh.feed(h2[a:a + n]))
            assert np.abs(np.concatenate(got) - want).max() < 3e-5 * max(1.0, np.abs(want).max()), (expand_over, portions)
            assert np.abs(np.concatenate(got2) - want2).max() < 3e-5 * max(1.0, np.abs(want2).max()), (expand_over, portions)


@pytest.mark.parametrize("portions", [[700], [640] + [1] * 60, [256, 256, 188], [63, 1, 64, 1, 2, 569], [2] * 350])
@pytest.mark.parametrize("j_star", [0, 1, 63, 64, 257])
def test_a_key_far_away_is_seen_from_its_own_position_on_and_never_before(dev, portions, j_star):
    """One head.  Every query scores 0 with every key but the one at j_star, which it scores with 60: whoever sees j_star returns its value."""
    m = {"heads": 1, "dim": 2, "rot_dim": 2, "vdim": 2, "kv_rank": 2, "scale": 1.0, "rot": {"dims": 2, "base": 10.0}}
    D, T = 4, 700
    w = {"m.q": np.zeros((4, D)), "m.g": np.zeros((1, D)), "m.dkv": np.eye(4, D), "m.dkv.norm": np.ones(2), "m.uk": np.zeros((2, 2)), "m.uv": np.eye(2), "m.o": np.eye(D, 2)}
    w["m.q"][0, 3] = 60.0 / np.sqrt(2.0)                       # a query reads the constant fourth column
    w["m.uk"][0, 1] = 1.0                                      # a key is its latent's second coordinate
    w["m.dkv"][3] = 0.0                                        # no rotated part: the fourth column does not reach the cache
    w["m.g"][0, 3] = 2.0
    h = np.zeros((T, D)); h[:, 0] = 1.0; h[:, 3] = 1.0
    h[j_star, :2] = (0.0, 1.0)
    o = feed_all(LatentMixer(dev, w, m, T, expand_over=8), h, portions)
    assert np.abs(o - R.latent_attention(h, R.latent_rows(h, w, "m.", m, 1e-5), w, "m.", m)).max() < 1e-4
    v = np.sqrt(2.0) * R.sigmoid(2.0)                          # the normed latent (0, sqrt 2), gated
    assert np.abs(o[:j_star, 1]).max(initial=0.0) < 1e-6       # nobody before it
    assert (np.abs(o[j_star:, 1] - v) < 1e-3).all() and np.abs(o[j_star:, 0]).max() < 1e-3


def test_rotated_halves_alone_find_a_key_by_its_distance(dev):
    """queries and keys agree only in ONE coordinate pair (i, i + 2) of the rotated part: the score is 1000 cos(i - j), largest at i = j; pairing
    neighbours instead would leave it 1000 everywhere (the partner of a lone coordinate would turn with another frequency)"""
    m = {"heads": 1, "dim": 1, "rot_dim": 4, "vdim": 1, "kv_rank": 1, "scale": 1000.0, "rot": {"dims": 4, "base": 1e8}}
    D, T = 3, 150
    w = {"m.q": np.zeros((5, D)), "m.g": np.zeros((1, D)), "m.dkv": np.zeros((5, D)), "m.dkv.norm": np.ones(1), "m.uk": np.zeros((1, 1)), "m.uv": np.ones((1, 1)), "m.o": np.eye(D, 1)}
    w["m.q"][1 + 2, 0] = w["m.dkv"][1 + 2, 0] = 1.0             # third rotated coordinate: partner of the first under halves, of the fourth under neighbours
    w["m.dkv"][0, 1] = 1.0
    h = np.zeros((T, D)); h[:, 0] = 1.0; h[:, 1] = np.where(np.arange(T) % 2, 1.0, -1.0)
    want = R.latent_attention(h, R.latent_rows(h, w, "m.", m, 1e-5), w, "m.", m)
    assert np.abs(want[:44, 0] - h[:44, 1] / 2).max() < 1e-3           # until seven full turns have passed every position returns its own value
    for portions in ([T], [100] + [1] * 50, [64, 1, 1, 84]):
        got = feed_all(LatentMixer(dev, w, m, T, expand_over=8), h, portions)
        assert np.abs(got - want).max() < 5e-3                         # scores of 1000 times a 32-bit cosine


def test_latent_ops_refuse_what_does_not_fit(dev):
    rng = np.random.default_rng(0)
    src, ring, f = T32(dev, rng.standard_normal((3, 20))), zeros(dev, 8, 6), T32(dev, [1.0])
    good = dict(q_src=src, q_col0=2, n_heads=2, dim=3, rest=2, freq=f, pairing=capi.ROPE_HALVES, mag=1.0, pos0=0, kv_src=src, kv_col0=14, ring=ring, norm_w=None, eps=1e-5)
    assert seqops.latent_prepare_append(**good).shape() == [3, 10]
    for bad in (dict(q_col0=11), dict(kv_col0=15), dict(ring=zeros(dev, 2, 6)), dict(ring=zeros(dev, 8, 2)), dict(norm_w=T32(dev, np.ones(3))), dict(freq=T32(dev, [1.0, 1.0])), dict(pairing=2)):
        with pytest.raises(capi.TensorError):
            seqops.latent_prepare_append(**dict(good, **bad))
    with pytest.raises(capi.TensorError):
        seqops.latent_query_append_paired(src, 2, T32(dev, rng.standard_normal((8, 3))), 2, 2, f, 7, 1.0, 0)
