"""CPU checks around the Nuvilorn decoder: the plain implementation against itself in other forms, the reader of model
folders, the registry, the layouts that are uploaded, and the trace runner's bookkeeping (a stand-in decoder)."""
import json
import struct

import numpy as np
import pytest

import nuvilorn_models as M
from oracle import nuvilorn as N


# ── the plain implementation ──
def test_folded_queries_give_the_same_attention():
    """(W_uk c) . q = c . (W_uk^T q): attention over the latents themselves, W_uv once at the end."""
    g = np.random.default_rng(3)
    mix = M.mixer(3, 10, 4, 6, 8, scale=0.7)
    n, W = 9, 12
    w = {"q": g.normal(size=(42, W)), "uk": g.normal(size=(30, 8)), "uv": g.normal(size=(18, 8)), "o": g.normal(size=(W, 18))}
    h, pos = g.normal(size=(n, W)), np.arange(n)
    c, kr = N.latent_of(h, pos, g.normal(size=(12, W)), g.uniform(0.5, 1.5, 8), mix, 1e-6)
    ref = N.latent_attention(h, pos, w, mix, (c, kr))
    q = (h @ w["q"].T).reshape(n, 3, 14)
    out = np.zeros((n, 18))
    for i in range(n):
        for hd in range(3):
            ql = q[i, hd, :10] @ w["uk"][hd * 10:hd * 10 + 10]
            qr = N.rotate_interleaved(q[i:i + 1, hd, 10:], [i], 4, mix["rot"]["base"])[0]
            s = (c[:i + 1] @ ql + kr[:i + 1] @ qr) * 0.7
            p = np.exp(s - s.max())
            out[i, hd * 6:hd * 6 + 6] = w["uv"][hd * 6:hd * 6 + 6] @ ((p / p.sum()) @ c[:i + 1])
    assert np.allclose(out @ w["o"].T, ref, rtol=1e-10, atol=1e-10)


def test_rotation_pairs_neighbours_and_depends_on_the_distance_only():
    g = np.random.default_rng(4)
    x, y = g.normal(size=6), g.normal(size=6)
    r = lambda v, p: N.rotate_interleaved(v[None], [p], 6, 100.0)[0]
    assert np.allclose(r(x, 7) @ r(y, 3), r(x, 104) @ r(y, 100))
    one = r(np.array([1.0, 0, 0, 0, 0, 0]), 2)
    assert np.allclose(one, [np.cos(2), np.sin(2), 0, 0, 0, 0])
    assert np.allclose(r(np.array([0, 0, 0, 1.0, 0, 0]), 1)[2:4], [-np.sin(100 ** (-1 / 3)), np.cos(100 ** (-1 / 3))])


def test_later_tokens_do_not_change_earlier_logits():
    cfg = M.CONFIGS["mixed"]
    w, t = M.weights(cfg), M.tokens(cfg, 20)
    full = N.forward(cfg, w, t)
    for n in (1, 2, 13):
        assert np.allclose(N.forward(cfg, w, t[:n]), full[:n], rtol=1e-9, atol=1e-9)


def test_the_weight_of_an_expert_multiplies_its_input():
    g = np.random.default_rng(5)
    h, up, down = g.normal(size=(1, 6)), g.normal(size=(4, 6)), g.normal(size=(6, 4))
    router = g.normal(size=(1, 6))
    s = N.sigmoid(h @ router.T)[0, 0]
    got = N.moe(h, {"router": router, "e0.up": up, "e0.down": down}, M.moe(4, 1, 1))
    assert np.allclose(got, s * s * N.relu2_ff(h, up, down)) and not np.allclose(got, s * N.relu2_ff(h, up, down))


# ── model folders ──
def test_safetensors_reader(tmp_path):
    from runit_mac_b200.safetensors import SafetensorsError, SafetensorsFile, bf16_to_f32, f32_to_bf16
    a = np.random.default_rng(0).normal(size=(3, 5)).astype(np.float32)
    kept = N.save_folder(tmp_path, {}, {"a": a, "s": np.array(2.0)})
    f = SafetensorsFile(tmp_path / "model.safetensors")
    assert f.shape("a") == (3, 5) and f.shape("s") == () and "b" not in f
    assert (f.f32("a") == kept["a"]).all() and f.f32("s") == 2.0
    assert (f.bf16("a") == N.to_bf16(a)).all() and (f32_to_bf16(a) == N.to_bf16(a)).all()
    assert (bf16_to_f32(f32_to_bf16(a)) == kept["a"]).all()
    with pytest.raises(SafetensorsError):
        f.tensor("b")
    head = json.dumps({"x": {"dtype": "BF16", "shape": [4], "data_offsets": [0, 6]}}).encode()
    (tmp_path / "bad").write_bytes(struct.pack("<Q", len(head)) + head + b"\0" * 8)
    with pytest.raises(SafetensorsError):
        SafetensorsFile(tmp_path / "bad")
    (tmp_path / "cut").write_bytes(struct.pack("<Q", 1000) + b"{}")
    with pytest.raises(SafetensorsError):
        SafetensorsFile(tmp_path / "cut")


class _Buf:
    def __init__(self, a):
        self.a, self.ptr = np.array(a), id(self)


class _Ctx:
    """Keeps what would be uploaded."""

    def __init__(self):
        self.bufs = {}

    def buffer_from(self, a):
        b = _Buf(a)
        self.bufs[b.ptr] = b.a
        return b


def _build(tmp_path, cfg, monkeypatch, dtype="bfloat16"):
    from runit_mac_b200 import dispatch, models
    w = M.folder(tmp_path, cfg)
    got = {}

    class Fake:
        def __init__(self, ctx, c, layers, ws, keep=()):
            got.update(ctx=ctx, cfg=c, layers=layers, w=ws)
    monkeypatch.setattr(dispatch, "LayeredModel", Fake)
    ctx = _Ctx()
    models.load_model(ctx, tmp_path, dtype, max_seq=64)
    return w, got, ctx.bufs


@pytest.mark.parametrize("name", sorted(M.CONFIGS))
def test_descriptors_and_layouts(tmp_path, monkeypatch, name):
    from runit_mac_b200 import dispatch as D
    cfg = M.CONFIGS[name]
    w, got, bufs = _build(tmp_path, cfg, monkeypatch, "float32")
    c = got["cfg"]
    assert (c.n_layers, c.width, c.vocab, c.max_seq, c.exact) == (len(cfg["layers"]), cfg["width"], cfg["vocab"], 64, 1)
    assert c.eps == np.float32(cfg["norm"]["eps"])
    W = cfg["width"]
    for i, (d, layer) in enumerate(zip(got["layers"], cfg["layers"])):
        m, f, p = layer["mixer"], layer["mlp"], "l%d." % i
        assert (d.heads, d.dim, d.rot_dim, d.vdim, d.kv_rank) == tuple(m[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
        assert d.scale == np.float32(m["scale"]) and d.rot_base == np.float32(m["rot"]["base"])
        q = N.from_bf16(bufs[d.w_q])
        assert q.shape[1] % 8 == 0 and (q[:, W:] == 0).all()
        own = m.get("kv_from") is None
        ref = np.concatenate([w[p + "mix.q"], w[p + "mix.dkv"]]) if own else w[p + "mix.q"]
        assert (q[:, :W] == ref).all() and d.kv_from == (-1 if own else m["kv_from"])
        assert bool(d.kv_norm) == own
        if f is None:
            assert d.ff_kind == D.FF_NONE and not d.norm2
        elif f["kind"] == "dense":
            u = N.from_bf16(bufs[d.ff_up])[:, :W]
            assert d.ff_kind == D.FF_DENSE and (u[0::2] == w[p + "mlp.gate"]).all() and (u[1::2] == w[p + "mlp.up"]).all()
        else:
            E = f["router"]["experts"]
            assert (d.ff_kind, d.n_experts, d.top_k, d.score, d.renorm) == (D.FF_MOE, E, f["router"]["top"], D.SCORE_SIGMOID, 0)
            down = N.from_bf16(bufs[d.ff_down]).reshape(E, W, -1)
            assert (down[E - 1, :, :f["expert"]["ff"]] == w[p + "mlp.e%d.down" % (E - 1)]).all()
            r = bufs[d.router].reshape(-1, W)
            assert len(r) == E + (1 if f.get("shared") else 0) and (r[:E] == w[p + "mlp.router"]).all()
            assert d.shared_ff == (f["shared"]["ff"] if f.get("shared") else 0)


def test_registry_refuses_what_it_does_not_know(tmp_path, monkeypatch):
    from runit_mac_b200 import models
    assert "Nuvilorn" in models.ARCHITECTURES
    base = M.CONFIGS["tiny"]
    for edit in (lambda c: c.update(architecture="Other"), lambda c: c["layers"][0].update(type="other"),
                 lambda c: c["layers"][0]["mlp"].update(kind="other"), lambda c: c["layers"][0]["mixer"].update(heads=2),
                 lambda c: c["layers"][0]["mixer"]["rot"].update(dims=4)):
        cfg = json.loads(json.dumps(base))
        M.folder(tmp_path, cfg)
        edit(cfg)
        (tmp_path / "config.json").write_text(json.dumps(cfg))
        with pytest.raises(models.ConfigError):
            models.load_model(_Ctx(), tmp_path)
    with pytest.raises(models.ConfigError):
        models.load_model(_Ctx(), tmp_path, dtype="int8")


# ── trace runner ──
class _Recorder:
    """Stand-in decoder: the logits of a token are (token, position)."""

    def __init__(self):
        self.calls = []

    def forward(self, tokens, start, want):
        self.calls.append((list(tokens), start))
        return np.array([[tokens[k], start + k] for k in want], np.float32).reshape(-1, 2)


def test_trace_replay(tmp_path):
    from runit_mac_b200 import trace
    m, said = _Recorder(), []
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [5, 6, 7], "want": [2, 0]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [8, 9], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": [4], "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": [3], "want": [0]}], "end": ["b"]}]
    trace.replay(m, [json.dumps(s) + "\n" for s in steps], tmp_path, said.append)
    assert said == ["done %d" % i for i in range(4)]
    assert m.calls == [([5, 6, 7], 0), ([8, 9], 3), ([4], 5), ([3], 0)]
    read = lambda i: np.fromfile(tmp_path / ("%d.f32" % i), "<f4").reshape(-1, 2).tolist()
    assert read(0) == [[7, 2], [5, 0]] and read(2) == [[4, 5]] and read(3) == [[3, 0]]
    assert not (tmp_path / "1.f32").exists()
    with pytest.raises(ValueError):
        trace.replay(m, [json.dumps(steps[0]), json.dumps(steps[3])], tmp_path, said.append)


def test_the_parts_of_the_library_name_existing_sources():
    from runit_mac_b200 import build
    for lib, names in build.PARTS.values():
        assert lib.suffix == ".so" and all((build.CSRC / (n + ".cu")).exists() for n in names)
