"""CPU checks around the Pagazen decoder: the plain implementation against itself in other forms, the registry and the layouts
that are uploaded."""
import json

import numpy as np
import pytest

import pagazen_models as M
from oracle import pagazen as P
from oracle.nuvilorn import from_bf16


# ── the plain implementation ──
def test_recurrence_in_chunks_gives_the_same():
    """Starting state times decays, plus the masked products within the chunk."""
    g = np.random.default_rng(1)
    n, H, dk, dv, C = 23, 2, 5, 4, 6
    q, k, v, a = g.normal(size=(n, H, dk)), g.normal(size=(n, H, dk)), g.normal(size=(n, H, dv)), g.uniform(0.3, 1.0, (n, H))
    ref = P.linear_scan(q, k, v, a)
    la, S, out = np.log(a), np.zeros((H, dk, dv)), np.zeros((n, H, dv))
    for t0 in range(0, n, C):
        t1 = min(n, t0 + C)
        c = np.cumsum(la[t0:t1], 0)
        for h in range(H):
            w = np.tril(np.exp(c[:, None, h] - c[None, :, h]))
            out[t0:t1, h] = np.exp(c[:, h, None]) * (q[t0:t1, h] @ S[h]) + (w * (q[t0:t1, h] @ k[t0:t1, h].T)) @ v[t0:t1, h]
            S[h] = np.exp(c[-1, h]) * S[h] + (k[t0:t1, h] * np.exp(c[-1, h] - c[:, h, None])).T @ v[t0:t1, h]
    assert np.allclose(out, ref, rtol=1e-10, atol=1e-10)


def test_window_and_bias():
    m = P.window_mask(6, 3)
    assert m.sum(1).tolist() == [1, 2, 3, 3, 3, 3] and m[5].tolist() == [False, False, False, True, True, True]
    assert np.allclose(P.head_slopes(8), [0.5, 0.25, 0.125, 0.0625, 2 ** -5, 2 ** -6, 2 ** -7, 2 ** -8]) and P.head_slopes(1) == 2 ** -8
    q = np.ones((4, 1, 2))
    s = P.biased_scores(q, q, 0.5, [0.25])[0]
    assert s[3, 1] == 1.0 - 0.5 and s[2, 2] == 1.0


def test_rotation_pairs_halves_and_depends_on_the_distance_only():
    g = np.random.default_rng(4)
    x, y = g.normal(size=8), g.normal(size=8)
    r = lambda v, p: P.rotate_halves(v[None, None], [p], 6, 100.0)[0, 0]
    assert np.allclose(r(x, 7) @ r(y, 3), r(x, 104) @ r(y, 100))
    one = r(np.eye(8)[0], 2)
    assert np.allclose(one, [np.cos(2), 0, 0, np.sin(2), 0, 0, 0, 0])
    assert np.allclose(r(np.eye(8)[4], 1), np.eye(8)[4] * np.cos(100 ** (-1 / 3)) - np.eye(8)[1] * np.sin(100 ** (-1 / 3)))
    assert (r(np.eye(8)[7], 9) == np.eye(8)[7]).all()


def test_convolution_looks_back_and_its_last_tap_is_the_current_token():
    x = np.zeros((5, 1))
    x[1] = 1.0
    y = P.causal_conv(x, np.array([[3.0, 2.0, 1.0]]), np.array([0.5]))
    assert y[:, 0].tolist() == [0.5, 1.5, 2.5, 3.5, 0.5]


@pytest.mark.parametrize("name", sorted(M.CONFIGS))
def test_later_tokens_do_not_change_earlier_logits(name):
    cfg = M.CONFIGS[name]
    w, t = M.weights(cfg), M.tokens(cfg, 40)
    full = P.forward(cfg, w, t)
    for n in (1, 2, 23):
        assert np.allclose(P.forward(cfg, w, t[:n]), full[:n], rtol=1e-9, atol=1e-9)
    assert np.abs(full).max() <= cfg["logit_softcap"] and full.std() > 0.1


# ── loading ──
class _Buf:
    def __init__(self, a):
        self.a, self.ptr = np.array(a), id(self)


class _Ctx:
    """Keeps what would be uploaded."""

    def __init__(self):
        self.bufs, self.keep = {}, []

    def buffer_from(self, a):
        b = _Buf(a)
        self.keep.append(b)
        self.bufs[b.ptr] = b.a
        return b


@pytest.mark.parametrize("name", sorted(M.CONFIGS))
def test_descriptors_and_layouts(tmp_path, monkeypatch, name):
    from runit_mac_b200 import dispatch as D, models
    cfg, got = M.CONFIGS[name], {}
    w = M.folder(tmp_path, cfg)

    class Fake:
        def __init__(self, ctx, c, layers, ws, keep=()):
            got.update(cfg=c, layers=layers, w=ws)
    monkeypatch.setattr(D, "LayeredModel", Fake)
    ctx = _Ctx()
    models.load_model(ctx, tmp_path, "float32", max_seq=64)
    c, bufs, W = got["cfg"], ctx.bufs, cfg["width"]
    assert (c.n_layers, c.width, c.vocab, c.max_seq, c.exact, c.post_norm) == (len(cfg["layers"]), W, cfg["vocab"], 64, 1, 1)
    assert c.eps == np.float32(cfg["norm"]["eps"]) and c.embed_scale == cfg["embedding"]["scale"] and c.logit_cap == cfg["logit_softcap"]
    assert (bufs[got["w"]["final_norm"]] == 1 + w["final.norm"]).all() and not got["w"].get("embed_norm")
    for i, (d, layer) in enumerate(zip(got["layers"], cfg["layers"])):
        if "weights_of" in layer:
            assert d is got["layers"][layer["weights_of"]]
            continue
        p, m = "l%d." % i, layer["mixer"]
        w_in, w_out = (from_bf16(bufs[x]) for x in (d.w_q, d.w_o))
        assert w_in.shape[1] % 8 == 0 and (w_in[:, W:] == 0).all() and (bufs[d.norm1] == 1 + w[p + "norm1"]).all()
        if layer["type"] == "parallel":
            a, r = m["left"], m["right"]
            assert d.mixer == D.MIX_HEADS and (d.at_heads, d.at_kv_heads, d.at_dim, d.at_vdim, d.at_window, d.at_unit_qk) == (
                a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["mask"]["size"], 1)
            assert (d.rt_heads, d.rt_dim, d.rt_vdim, d.rt_rot_dims) == (r["heads"], r["dim"], r["vdim"], r["rot"]["dims"])
            assert (d.at_out_scale, d.rt_out_scale) == (np.float32(m["left_scale"]), np.float32(m["right_scale"])) and d.at_scale == np.float32(a["scale"])
            assert np.allclose(bufs[d.at_slopes], P.head_slopes(a["heads"])) and np.allclose(bufs[d.rt_decay][0], r["decay"])
            assert np.allclose(np.exp(bufs[d.rt_decay][1]), r["decay"])
            ref = np.concatenate([w[p + "mix.left." + n] for n in "qkv"] + [w[p + "mix.right." + n] for n in "qkvg"])
            out = np.concatenate([w[p + "mix.left.o"], w[p + "mix.right.o"]], 1)
        else:
            assert d.mixer == D.MIX_SSM and (d.ss_heads, d.ss_vdim, d.ss_state, d.ss_groups, d.ss_taps, d.ss_norm_groups) == tuple(
                m[k] for k in ("heads", "vdim", "state", "groups", "conv", "norm_groups"))
            assert np.allclose(bufs[d.ss_a], -np.exp(w[p + "mix.A_log"])) and (bufs[d.ss_conv].reshape(-1, m["conv"]) == w[p + "mix.conv"]).all()
            ref, out = w[p + "mix.in"], w[p + "mix.o"]
        assert (w_in[:, :W] == ref).all() and (w_out[:, :out.shape[1]] == out).all() and (w_out[:, out.shape[1]:] == 0).all()
        if layer["mlp"] is None:
            assert d.ff_kind == D.FF_NONE and not d.norm2
        else:
            assert (d.ff_kind, d.ff_act, d.ff) == (D.FF_DENSE, D.ACT_RELU2, layer["mlp"]["ff"])


def test_a_decay_of_zero_has_a_finite_logarithm(tmp_path, monkeypatch):
    from runit_mac_b200 import dispatch as D, models
    cfg, got = M.config(16, 20, [(M.parallel(M.left(1, 1, 8, 8, 4), M.right(2, 8, 8, 8, decay=[0.0, 0.75])), 8)]), {}
    M.folder(tmp_path, cfg)
    monkeypatch.setattr(D, "LayeredModel", lambda ctx, c, layers, ws, keep=(): got.update(d=layers[0]))
    ctx = _Ctx()
    models.load_model(ctx, tmp_path)
    dec = ctx.bufs[got["d"].rt_decay]
    assert dec[0].tolist() == [0.0, 0.75] and np.isfinite(dec).all() and np.exp(dec[1, 0]) == 0 and np.float32(128) * dec[1, 0] > -1e30


def test_registry_refuses_what_it_does_not_know(tmp_path):
    from runit_mac_b200 import models
    base = M.config(16, 20, [(M.parallel(M.left(2, 1, 8, 8, 4), M.right(2, 8, 8, 8)), 8), (M.mamba(2, 8, 8), 8), 0])

    def change(path, value):
        def edit(c):
            for k in path[:-1]:
                c = c[k]
            c[path[-1]] = value
        return edit
    for edit in (change(("layers", 0, "type"), "other"), change(("layers", 0, "mlp", "kind"), "other"), change(("layers", 0, "mixer", "left", "heads"), 4),
                 change(("layers", 0, "mixer", "right", "decay"), [0.5]), change(("layers", 1, "mixer", "state"), 16), change(("layers", 1, "mixer", "conv"), 3),
                 change(("layers", 2, "weights_of"), 5), change(("layers", 2, "weights_of"), 1), change(("width",), 24)):
        cfg = json.loads(json.dumps(base))
        M.folder(tmp_path, cfg)
        edit(cfg)
        (tmp_path / "config.json").write_text(json.dumps(cfg))
        with pytest.raises(models.ConfigError):
            models.load_model(_Ctx(), tmp_path)
