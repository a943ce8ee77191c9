"""GPU tests of the Nuvilorn decoder and the mechanisms it is made of, against the plain implementation (oracle/nuvilorn.py)."""
import ctypes as C

import numpy as np
import pytest

import nuvilorn_models as M
from oracle import nuvilorn as N

pytestmark = pytest.mark.gpu

EXACT = 3e-5         # row error (relative to the spread of the logits) in 32-bit


def bf16_rows(a):
    """bf16 bit patterns with rows padded to multiples of 8, and the values they hold."""
    a = np.asarray(a, np.float32)
    u = np.zeros(a.shape[:-1] + ((a.shape[-1] + 7) // 8 * 8,), np.uint16)
    u[..., :a.shape[-1]] = N.to_bf16(a).reshape(a.shape)
    return u, N.from_bf16(u)[..., :a.shape[-1]].astype(np.float64)


def close(got, ref, tol):
    """Within tol of the larger of the value itself and the root mean square."""
    got, ref = np.asarray(got, np.float64), np.asarray(ref, np.float64)
    assert np.isfinite(got).all()
    err = (np.abs(got - ref) / np.maximum(np.abs(ref), max(np.sqrt((ref ** 2).mean()), 1e-30))).max()
    assert err <= tol, err


# ── mechanisms ──
@pytest.mark.parametrize("T,width", [(1, 8), (3, 100), (5, 1000), (2, 2048)])
def test_norm_with_one_gain(ctx, T, width):
    import runit_mac_b200 as R
    g = np.random.default_rng(T)
    x = (g.normal(size=(T, width)) * np.array([10.0 ** -i for i in range(T)])[:, None]).astype(np.float32)   # eps matters in the small rows
    gain = np.array([1.37], np.float32)
    ld = (width + 7) // 8 * 8
    for f32 in (1, 0):
        y = ctx.new_buffer(T * ld * 4)
        R.norm_gain_rows(ctx, ctx.buffer_from(x), ctx.buffer_from(gain), 1e-3, y, f32, T, width)
        ctx.flush()
        got = y.download(np.float32, T * ld) if f32 else N.from_bf16(y.download(np.uint16, T * ld))
        got = got.reshape(T, ld)
        ref = N.rms_norm_scalar(x.astype(np.float64), gain, 1e-3)
        assert (got[:, width:] == 0).all()
        for t in range(T):
            close(got[t, :width], ref[t], 1e-6 * 5 if f32 else 2e-2)


@pytest.mark.parametrize("m,k", [(1, 8), (7, 20), (65, 300), (200, 1000), (333, 1032), (64, 2500), (4, 12000)])
def test_gemv(ctx, m, k):
    import runit_mac_b200 as R
    g = np.random.default_rng(m)
    u, w = bf16_rows(g.normal(size=(m, k)))
    x, r, gain = g.normal(size=k).astype(np.float32), g.normal(size=m).astype(np.float32), np.array([0.8], np.float32)
    wb, xb, y = ctx.buffer_from(u), ctx.buffer_from(x), ctx.new_buffer(m * 4)
    R.gemv_bf16_f32(ctx, wb, xb, None, 0.0, y, ctx.buffer_from(r), m, k)
    ctx.flush()
    close(y.download(np.float32, m), w @ x.astype(np.float64) + r, 1e-5)
    R.gemv_bf16_f32(ctx, wb, xb, ctx.buffer_from(gain), 1e-2, y, None, m, k)
    ctx.flush()
    close(y.download(np.float32, m), w @ N.rms_norm_scalar(x.astype(np.float64), gain, 1e-2), 1e-5)


@pytest.mark.parametrize("T,m,k", [(1, 2, 8), (2, 130, 40), (17, 64, 100), (70, 300, 200), (200, 258, 96), (513, 128, 64), (300, 1030, 520),
                                   (900, 4096, 256), (64, 20000, 72)])
def test_gemm(ctx, T, m, k):
    """Both kernels with every epilogue."""
    import runit_mac_b200 as R
    g = np.random.default_rng(T)
    u, w = bf16_rows(g.normal(size=(m, k)) / np.sqrt(k))
    xu, xv = bf16_rows(g.normal(size=(T, k)))
    ld = xu.shape[1]
    xf = np.zeros((T, ld), np.float32)
    xf[:, :k] = xv
    pre, post = g.uniform(0.2, 2, T).astype(np.float32), g.uniform(0.2, 2, T).astype(np.float32)
    wb, pb, qb = ctx.buffer_from(u), ctx.buffer_from(pre), ctx.buffer_from(post)
    z = xv @ w.T
    base = g.normal(size=(T, m)).astype(np.float32)
    zp = z * pre[:, None]
    refs = {R.EPI_F32: z, R.EPI_ADD: z + base, R.EPI_CAST: z, R.EPI_RELU2: np.maximum(zp, 0) ** 2 * post[:, None],
            R.EPI_SILU_GLU: zp[:, 0::2] * N.sigmoid(zp[:, 0::2]) * zp[:, 1::2] * post[:, None]}
    for exact in (1, 0):
        xb = ctx.buffer_from(xf if exact else xu)
        for epi, ref in refs.items():
            y = ctx.buffer_from(base) if epi == R.EPI_ADD else ctx.new_buffer(max(T * m * 4, 16))
            n = ref.shape[1]
            act = epi >= R.EPI_SILU_GLU
            R.gemm_bf16_rows(ctx, wb, xb, y, n, T, m, k, exact, epi, pb if act else None, qb if act else None)
            ctx.flush()
            f32 = exact or epi in (R.EPI_F32, R.EPI_ADD)
            got = y.download(np.float32, T * n) if f32 else N.from_bf16(y.download(np.uint16, T * n))
            close(got.reshape(T, n), ref, 3e-5 if f32 else 1e-2)


def test_gemm_repeats_bit_for_bit(ctx):
    import runit_mac_b200 as R
    g = np.random.default_rng(0)
    u, _ = bf16_rows(g.normal(size=(384, 256)))
    xu, _ = bf16_rows(g.normal(size=(600, 256)))
    wb, xb = ctx.buffer_from(u), ctx.buffer_from(xu)
    outs = []
    for _ in range(3):
        y = ctx.new_buffer(600 * 384 * 4)
        R.gemm_bf16_rows(ctx, wb, xb, y, 384, 600, 384, 256, 0, R.EPI_F32, None, None)
        ctx.flush()
        outs.append(y.download(np.uint32, 600 * 384))
    assert (outs[0] == outs[1]).all() and (outs[0] == outs[2]).all()


@pytest.mark.parametrize("E,k,ld", [(1, 1, 2), (5, 3, 6), (40, 8, 40), (100, 2, 101), (256, 32, 256)])
def test_sigmoid_routing(ctx, E, k, ld):
    import runit_mac_b200 as R
    g = np.random.default_rng(E)
    T = 9
    z = g.normal(0, 3, (T, ld)).astype(np.float32)
    z[:, E:] = 50.0                                   # columns past the experts never win
    z[0, :E] = 20.0 + g.permutation(E) * 0.01        # scores that all round to 1: the logits decide
    idx, w = ctx.new_buffer(T * k * 4), ctx.new_buffer(T * k * 4)
    R.moe_route_scored(ctx, ctx.buffer_from(z), ld, E, k, R.SCORE_SIGMOID, 0, T, idx, w)
    ctx.flush()
    ref = np.argsort(-z[:, :E].astype(np.float64), axis=1, kind="stable")[:, :k]
    got = idx.download(np.int32, T * k).reshape(T, k)
    assert (got == ref).all()
    assert np.allclose(w.download(np.float32, T * k).reshape(T, k), N.sigmoid(np.take_along_axis(z, ref, 1).astype(np.float64)), rtol=2e-6)


def _latent_case(mix, T, start, seed, f32, spike=None):
    """Random projections of `start + T` positions; returns inputs and the plain result for the last T."""
    g = np.random.default_rng(seed)
    H, d, r, dv, rank = (mix[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    n = start + T
    raw = g.normal(size=(n, rank + r)).astype(np.float32)
    q = g.normal(size=(n, H * (d + r))).astype(np.float32)
    if spike is not None:                             # a query whose scores stand out
        q[spike] *= 3.0
    kvn = g.uniform(0.5, 1.5, rank).astype(np.float32)
    uk_u, uk = bf16_rows(g.normal(size=(H * d, rank)) / np.sqrt(rank))
    uv_u, uv = bf16_rows(g.normal(size=(H * dv, rank)) / np.sqrt(rank))
    pos = np.arange(n)
    c = N.rms_norm(raw[:, :rank].astype(np.float64), kvn, 1e-5)
    kr = N.rotate_interleaved(raw[:, rank:].astype(np.float64), pos, r, mix["rot"]["base"])
    if not f32:
        c, kr = N.from_bf16(N.to_bf16(c)).reshape(c.shape).astype(np.float64), N.from_bf16(N.to_bf16(kr)).reshape(kr.shape).astype(np.float64)
    qq = q.reshape(n, H, d + r).astype(np.float64)
    q_rot = N.rotate_interleaved(qq[..., d:], pos, r, mix["rot"]["base"])
    s = np.einsum("ihd,jhd->hij", qq[..., :d], (c @ uk.T).reshape(n, H, d)) + np.einsum("ihd,jd->hij", q_rot, kr)
    p = N.causal_softmax(s * mix["scale"])
    out = np.einsum("hij,jhd->ihd", p, (c @ uv.T).reshape(n, H, dv)).reshape(n, H * dv)
    return raw, q, kvn, uk_u, uv_u, out[start:], p[:, start:, :]


LATENT = [(M.mixer(3, 24, 8, 40, 48), 5, 0), (M.mixer(16, 128, 64, 128, 512), 1, 700), (M.mixer(20, 32, 16, 33, 100), 7, 130),
          (M.mixer(5, 7, 2, 9, 11), 40, 3), (M.mixer(2, 48, 32, 64, 1000), 3, 65), (M.mixer(1, 16, 8, 8, 16), 130, 0)]


@pytest.mark.parametrize("case", range(len(LATENT)))
@pytest.mark.parametrize("f32", [1, 0])
@pytest.mark.parametrize("nsplit", [1, 3, 64])
def test_folded_attention(ctx, case, f32, nsplit):
    import runit_mac_b200 as R
    mix, T, start = LATENT[case]
    raw, q, kvn, uk, uv, ref, _ = _latent_case(mix, T, start, case, f32)
    H, d, r, dv, rank = (mix[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    n, cp = start + T, (rank + 15) // 16 * 16
    pitch, ldq = cp + (r + 15) // 16 * 16, H * (d + r) + rank + r
    cfg = R.LatentCfg(H, d, r, dv, rank, mix["scale"], 1e-5)
    freq = ctx.buffer_from((mix["rot"]["base"] ** (-2.0 * np.arange(r // 2) / r)).astype(np.float32))
    qkv = np.concatenate([q, raw], 1)
    es = 4 if f32 else 2
    cache = ctx.buffer_from(np.zeros(n * pitch * es, np.uint8))
    ukb, uvb, kb = ctx.buffer_from(uk), ctx.buffer_from(uv), ctx.buffer_from(kvn)
    if start:      # earlier positions: their rows only, in portions
        R.latent_rows(ctx, C.byref(cfg), f32, ctx.buffer_from(qkv[:start]), ldq, kb, freq, cache, start, 0)
    qe = ctx.new_buffer(T * H * pitch * 4)
    R.latent_query(ctx, C.byref(cfg), f32, ctx.buffer_from(qkv[start:]), ldq, ukb, kb, freq, cache, qe, T, start)
    po, ml, out = ctx.new_buffer(T * H * nsplit * cp * 4), ctx.new_buffer(T * H * nsplit * 8), ctx.new_buffer(T * H * dv * 4)
    R.latent_attention(ctx, C.byref(cfg), f32, qe, cache, po, ml, nsplit, T, start)
    R.latent_value(ctx, C.byref(cfg), po, ml, nsplit, uvb, out, T)
    ctx.flush()
    close(out.download(np.float32, T * H * dv).reshape(T, H * dv), ref, 2e-5 if f32 else 2e-2)


@pytest.mark.parametrize("H,d,r,dv,rank,T,start", [(2, 24, 8, 40, 48, 70, 0), (3, 64, 32, 56, 72, 129, 50), (2, 96, 32, 64, 40, 65, 64),
                                                   (2, 64, 64, 128, 80, 200, 1), (2, 128, 64, 128, 512, 150, 37), (1, 8, 8, 8, 16, 64, 63)])
def test_expanded_attention(ctx, H, d, r, dv, rank, T, start):
    import runit_mac_b200 as R
    mix = M.mixer(H, d, r, dv, rank, scale=0.5)
    # the last query points sharply at its keys: a key that is dropped or let in shows
    raw, q, kvn, uk, uv, _, _ = _latent_case(mix, T, start, T, 0, spike=start + T - 1)
    n, cp = start + T, (rank + 15) // 16 * 16
    pitch, ldq = cp + (r + 15) // 16 * 16, H * (d + r) + rank + r
    cfg = R.LatentCfg(H, d, r, dv, rank, 0.5, 1e-5)
    freq = ctx.buffer_from((mix["rot"]["base"] ** (-2.0 * np.arange(r // 2) / r)).astype(np.float32))
    qkv = ctx.buffer_from(np.concatenate([q, raw], 1))
    cache, kb = ctx.buffer_from(np.zeros(n * pitch, np.uint16)), ctx.buffer_from(kvn)
    R.latent_rows(ctx, C.byref(cfg), 0, qkv, ldq, kb, freq, cache, n, 0)
    ctx.flush()
    lat = N.from_bf16(cache.download(np.uint16, n * pitch)).reshape(n, pitch)[:, :rank].astype(np.float64)
    ukv = np.concatenate([uk, uv]).astype(np.uint16)
    w = N.from_bf16(ukv)[:, :rank].astype(np.float64)
    kv, kvv = bf16_rows(lat @ w.T)
    ldo = (H * dv + 7) // 8 * 8
    out = ctx.new_buffer(T * ldo * 2)
    R.latent_prefill_attention(ctx, C.byref(cfg), qkv.ptr + start * ldq * 4, ldq, ctx.buffer_from(kv), kv.shape[1], cache, out, ldo, T, start)
    ctx.flush()
    # the plain result from the same expanded keys and values
    rows = N.from_bf16(cache.download(np.uint16, n * pitch)).reshape(n, pitch).astype(np.float64)
    qq = q.reshape(n, H, d + r).astype(np.float64)
    q_rot = N.rotate_interleaved(qq[..., d:], np.arange(n), r, mix["rot"]["base"])
    s = np.einsum("ihd,jhd->hij", qq[..., :d], kvv[:, :H * d].reshape(n, H, d)) + np.einsum("ihd,jd->hij", q_rot, rows[:, cp:cp + r])
    ref = np.einsum("hij,jhd->ihd", N.causal_softmax(s * 0.5), kvv[:, H * d:].reshape(n, H, dv)).reshape(n, H * dv)[start:]
    close(N.from_bf16(out.download(np.uint16, T * ldo)).reshape(T, ldo)[:, :H * dv], ref, 6e-2)


# ── the model ──
class Served:
    def __init__(self, ctx, path, cfg, dtype, max_seq=320, **kw):
        from runit_mac_b200 import models
        self.cfg, self.w = cfg, M.folder(path, cfg, **kw)
        self.m = models.load_model(ctx, path, dtype, max_seq)

    def run(self, tokens, cuts, want=None):
        """Logits of `want` (default: all) with the tokens cut into portions of the given sizes (repeating)."""
        want = range(len(tokens)) if want is None else want
        out, pos, i = [], 0, 0
        while pos < len(tokens):
            c = min(cuts[i % len(cuts)], len(tokens) - pos)
            i += 1
            out.append(self.m.forward(tokens[pos:pos + c], pos, [p - pos for p in want if pos <= p < pos + c]))
            pos += c
        return np.concatenate(out)


@pytest.fixture(params=["float32", "bfloat16"])
def dtype(request):
    return request.param


def check_rows(got, ref, dtype, margins=None):
    """margins (bf16): tokens whose routing is a close call may go to another expert than in the plain implementation."""
    e = M.row_errors(got, ref)
    if dtype == "float32":
        assert e.max() <= EXACT, e.max()
        return
    clear = e if margins is None else e[margins[:len(e)] > 0.2]
    if len(clear):
        assert np.median(clear) <= 0.02 and (clear > 0.08).mean() <= 0.02, (np.median(clear), np.sort(clear)[-5:])


@pytest.mark.parametrize("name", sorted(M.CONFIGS))
@pytest.mark.parametrize("n", [1, 2, 31, 32, 150])
def test_prompt(ctx, tmp_path, dtype, name, n):
    s = Served(ctx, tmp_path, M.CONFIGS[name], dtype)
    t = M.tokens(s.cfg, n)
    check_rows(s.run(t, [n]), N.forward(s.cfg, s.w, t), dtype, M.routing_margins(s.cfg, s.w, t))


@pytest.mark.parametrize("name", sorted(M.CONFIGS))
def test_prefill_against_token_by_token_and_portions(ctx, tmp_path, dtype, name):
    s = Served(ctx, tmp_path, M.CONFIGS[name], dtype, gain=2.0)
    t = M.tokens(s.cfg, 100)
    ref, mg = N.forward(s.cfg, s.w, t), M.routing_margins(s.cfg, s.w, t)
    whole = s.run(t, [100])
    for cuts in ([1], [2], [3, 2], [31, 1, 33], [64, 36], [99, 1], [7, 50, 2]):
        check_rows(s.run(t, cuts), ref, dtype, mg)
    if dtype == "float32":
        assert M.row_errors(s.run(t, [1]), whole).max() <= EXACT


def test_layer_by_layer(ctx, tmp_path):
    s = Served(ctx, tmp_path, M.CONFIGS["mixed"], "float32")
    t = M.tokens(s.cfg, 45)
    _, trail = N.forward(s.cfg, s.w, t, want_layers=True)
    s.m.set_depth(0)
    s.m.forward(t, 0)
    close(s.m.residual(45), N.rms_norm_scalar(np.asarray(s.w["embed"], np.float64)[t], s.w["embed.norm"], 1e-5), 1e-5)
    for d in range(1, len(trail) + 1):
        s.m.set_depth(d)
        s.m.forward(t, 0)
        close(s.m.residual(45), trail[d - 1], 3e-5)


ALONE = {
    "attention": M.config(48, 60, [(M.mixer(3, 16, 8, 24, 32), None)]),
    "borrowed latent": M.config(48, 60, [(M.mixer(3, 16, 8, 24, 32), None), (M.mixer(2, 24, 8, 16, 32, kv_from=0), None)]),
    "dense": M.config(48, 60, [(M.mixer(1, 8, 2, 8, 8), M.dense(40))]),
    "experts": M.config(48, 60, [(M.mixer(1, 8, 2, 8, 8), M.moe(24, 9, 4))]),
    "one expert of many": M.config(48, 60, [(M.mixer(1, 8, 2, 8, 8), M.moe(24, 9, 1))]),
    "experts and shared": M.config(48, 60, [(M.mixer(1, 8, 2, 8, 8), M.moe(24, 4, 2, 72))]),
}


@pytest.mark.parametrize("name", sorted(ALONE))
def test_mechanism_alone(ctx, tmp_path, dtype, name):
    """One mechanism per model: where the feed-forward is looked at, the output projection of the attention is zero."""
    cfg = ALONE[name]

    def edit(w):
        if cfg["layers"][0]["mlp"] is not None:
            w["l0.mix.o"][:] = 0
    s = Served(ctx, tmp_path, cfg, dtype, edit=edit)
    t = M.tokens(cfg, 60)
    ref, mg = N.forward(cfg, s.w, t), M.routing_margins(cfg, s.w, t)
    check_rows(s.run(t, [60]), ref, dtype, mg)
    check_rows(s.run(t, [1]), ref, dtype, mg)


def _only(monkeypatch, name, fault):
    monkeypatch.setattr(N, name, fault(getattr(N, name)))


FAULTS = {
    "a far key dropped": ("causal_softmax", lambda f: lambda s: _drop(f, s, 3)),
    "the first key dropped": ("causal_softmax", lambda f: lambda s: _drop(f, s, 0)),
    "the next key let in": ("causal_softmax", lambda f: lambda s: _peek(s)),
    "halves rotated instead of neighbours": ("rotate_interleaved", lambda f: lambda x, p, d, b: _halves(f, x, p, d, b)),
    "positions off by one in the query": ("rotate_interleaved", lambda f: lambda x, p, d, b: f(x, np.asarray(p) + (x.ndim == 3), d, b)),
    "the weight on the expert's output": ("moe", lambda f: lambda h, w, m: _weight_outside(h, w, m)),
    "latent not normed": ("rms_norm", lambda f: lambda x, w, e: x * w),
}


def _drop(f, s, j):
    s = np.array(s)
    s[..., 40:, j] = -1e9
    return f(s)


def _peek(s):
    n = s.shape[-1]
    s = np.where(np.arange(n)[None, :] <= np.arange(n)[:, None] + 1, s, -np.inf)
    p = np.exp(s - s.max(-1, keepdims=True))
    return p / p.sum(-1, keepdims=True)


def _halves(f, x, p, d, b):
    order = np.concatenate([np.arange(0, d // 2)[:, None], np.arange(d // 2, d)[:, None]], 1).reshape(-1)
    return f(x[..., order], p, d, b)


def _weight_outside(h, w, m):
    idx, sc = N.route_sigmoid(h, w["router"], m["router"]["top"])
    out = np.zeros_like(h)
    for t in range(len(h)):
        for e, a in zip(idx[t], sc[t]):
            out[t] += a * N.relu2_ff(h[t], w["e%d.up" % e], w["e%d.down" % e])
    if m.get("shared"):
        out += N.sigmoid(h @ w["shared.sg"].T) * N.relu2_ff(h, w["shared.up"], w["shared.down"])
    return out


def test_faults_would_show(ctx, tmp_path, monkeypatch):
    """Peaked attention (scores scaled up) makes single keys count.  A mistake in the plain implementation moves its logits
    far beyond the tolerances above, away from what the decoder computes in prompts and in decoding."""
    cfg = M.config(96, 131, [(M.mixer(4, 32, 16, 32, 48), M.moe(40, 6, 2, 56)), (M.mixer(3, 24, 16, 40, 48, kv_from=0), M.dense(64))])
    s = Served(ctx, tmp_path, cfg, "float32", gain=5.0)
    t = M.tokens(cfg, 80)
    prompt, decoded = s.run(t, [80]), s.run(t, [40] + [1] * 40)
    ref = N.forward(cfg, s.w, t)
    assert max(M.row_errors(prompt, ref).max(), M.row_errors(decoded, ref).max()) <= 10 * EXACT
    for what, (name, fault) in FAULTS.items():
        with monkeypatch.context() as mp:
            _only(mp, name, fault)
            bad = N.forward(cfg, s.w, t)
        for got in (prompt, decoded):
            e = M.row_errors(got, bad)
            assert e[40:].max() > 0.02 and e[40:].max() > 100 * EXACT, (what, e[40:].max())


@pytest.mark.parametrize("far", [0, 1, 63, 64, 127, 128, 200])
def test_one_key_far_away(ctx, tmp_path, dtype, far):
    """One token has a latent and a key part of its own that a marked query looks for: almost all weight goes to a position at
    a block's edge or at the start, hundreds of tokens back, in a prompt, in a short portion and in decoding."""
    cfg = M.config(64, 40, [(M.mixer(2, 32, 8, 32, 32, scale=0.6), None)])
    MARK, ASK = 38, 39

    def edit(w):
        u = np.zeros(64); u[0] = 8.0
        v = np.zeros(64); v[1] = 8.0
        w["embed"][:, :2] = 0
        w["embed"][MARK], w["embed"][ASK] = u, v
        w["l0.mix.dkv"][:, 0] = 0
        w["l0.mix.dkv"][:32, 0] = np.where(np.arange(32) == 5, 4.0, 0.0)      # the mark's latent is one coordinate
        w["l0.mix.dkv.norm"][:] = 1
        w["l0.mix.uk"][:, 5] = 0.5
        q = w["l0.mix.q"].reshape(2, 40, 64)
        q[:, :, 1] = 0
        q[:, :32, 1] = 0.6                                                    # the asking token looks for that coordinate
    s = Served(ctx, tmp_path, cfg, dtype, edit=edit)
    g = np.random.default_rng(far)
    t = [int(x) for x in g.integers(0, 38, 260)]
    t[far] = MARK
    t[255] = t[259] = ASK
    ref = N.forward(cfg, s.w, t)
    blind = [x for x in t]
    blind[far] = t[far - 1] if far else 7
    other = N.forward(cfg, s.w, blind)
    for p in (255, 259):
        assert M.row_errors(other[p:p + 1], ref[p:p + 1]).max() > 0.3          # the answer hangs on the marked token
    for cuts in ([260], [250, 10], [128, 127, 5], [200] + [1] * 60):
        got = s.run(t, cuts, want=[255, 259])
        assert M.row_errors(got, ref[[255, 259]]).max() <= (1e-4 if dtype == "float32" else 0.05)


def test_cache_is_reused_and_cut_back(ctx, tmp_path, dtype):
    """Another sequence after the first, a shorter one after a longer one, and a sequence taken up again from the middle."""
    s = Served(ctx, tmp_path, M.CONFIGS["mixed"], dtype)
    a, b = M.tokens(s.cfg, 120, 5), M.tokens(s.cfg, 50, 6)
    ra, mg = N.forward(s.cfg, s.w, a), lambda t: M.routing_margins(s.cfg, s.w, t)
    ma = mg(a)
    check_rows(s.run(a, [120]), ra, dtype, ma)
    check_rows(s.run(b, [20, 1, 29]), N.forward(s.cfg, s.w, b), dtype, mg(b))
    check_rows(s.run(a, [60, 1]), ra, dtype, ma)
    mixed = a[:40] + b[:30]
    got = s.m.forward(mixed[40:], 40, range(30))          # positions 40.. are overwritten
    check_rows(got, N.forward(s.cfg, s.w, mixed)[40:], dtype, mg(mixed)[40:])
    check_rows(s.run(a, [17]), ra, dtype, ma)


def test_long_prompt_is_cut_inside(ctx, tmp_path, dtype):
    """Prompts longer than one batched portion (256 tokens in 32-bit, 2048 in bf16)."""
    cfg = M.config(32, 60, [(M.mixer(2, 16, 8, 16, 16), M.dense(32)), (M.mixer(2, 16, 8, 16, 16, kv_from=0), M.moe(16, 4, 2, 8))])
    n = 600 if dtype == "float32" else 2150
    s = Served(ctx, tmp_path, cfg, dtype, max_seq=n + 8)
    t = M.tokens(cfg, n)
    want = [0, 255, 256, 511, 512, n - 1] if dtype == "float32" else [0, 2047, 2048, 2049, n - 1]
    ref = N.forward(cfg, s.w, t)
    got = s.run(t, [n], want=want)
    assert M.row_errors(got, ref[want]).max() <= (1e-4 if dtype == "float32" else 0.1)
    nxt = s.m.prefill(t)
    top = np.sort(ref[-1])[-2:]
    assert nxt == int(np.argmax(ref[-1])) or (dtype == "bfloat16" and top[1] - top[0] < 0.1 * np.std(ref[-1]))


def test_wanted_places_keep_their_order(ctx, tmp_path):
    s = Served(ctx, tmp_path, M.CONFIGS["mixed"], "float32")
    t = M.tokens(s.cfg, 90)
    ref = N.forward(s.cfg, s.w, t)
    want = [89, 3, 3, 40] + list(range(80, 0, -1))
    got = s.m.forward(t, 0, want)
    assert M.row_errors(got, ref[want]).max() <= EXACT
    assert s.m.forward(t[:5], 0, []).shape == (0, s.cfg["vocab"])


def test_greedy_generation(ctx, tmp_path):
    """Prefill and recorded decode steps, and the token-by-token path, give the plain implementation's continuation."""
    s = Served(ctx, tmp_path, M.CONFIGS["mixed"], "float32")
    p = M.tokens(s.cfg, 21)
    ref = M.greedy(s.cfg, s.w, p, 40)
    assert len(set(ref)) > 3
    assert s.m.generate(p, 40).tolist() == ref
    assert s.m.generate_greedy(p, 39)[len(p) - 1:].tolist() == ref
    assert s.m.prefill(p) == ref[0]
    seq, got = list(p), []
    for _ in range(5):
        got.append(s.m.forward_greedy(seq[-1], len(seq) - 1))
        seq.append(got[-1])
    assert got == ref[:5]
    # portions continue from where generation left the cache
    lg = s.m.forward(ref[4:8], len(p) + 4, [3])
    assert int(np.argmax(lg[0])) == ref[8]


def test_long_decoding(ctx, tmp_path, dtype):
    s = Served(ctx, tmp_path, M.CONFIGS["mixed"], dtype, max_seq=400)
    p = M.tokens(s.cfg, 3)
    out = s.m.generate_greedy(p, 380)[len(p) - 1:].tolist()
    seq = p + out
    ref = N.forward(s.cfg, s.w, seq[:-1])[len(p) - 1:]
    margin = np.sort(ref, 1)[:, -1] - ref[np.arange(len(out)), out]
    agree = (margin <= (1e-3 if dtype == "float32" else 0.25) * np.std(ref)).mean()
    assert agree == 1.0 if dtype == "float32" else agree > 0.95, agree


def test_sampled_generation(ctx, tmp_path):
    import runit_mac_b200 as R
    s = Served(ctx, tmp_path, M.CONFIGS["mixed"], "bfloat16")
    p = M.tokens(s.cfg, 12)
    a = s.m.generate_sampled(p, 30, R.SamplerCfg(0.9, 20, 0.95, 1.1, 0), seed=3)
    b = s.m.generate_sampled(p, 30, R.SamplerCfg(0.9, 20, 0.95, 1.1, 0), seed=3)
    c = s.m.generate_sampled(p, 30, R.SamplerCfg(0.9, 20, 0.95, 1.1, 0), seed=4)
    assert (a == b).all() and (a != c).any() and ((a[11:] >= 0) & (a[11:] < s.cfg["vocab"])).all()
    zero = s.m.generate_sampled(p, 30, R.SamplerCfg(0.0, 0, 1.0, 1.0, 0), seed=1)
    assert (zero[11:] == s.m.generate_greedy(p, 30)[11:]).all()


def test_command_line(ctx, tmp_path, capsys):
    from runit_mac_b200.__main__ import main
    cfg = M.CONFIGS["odd"]
    w = M.folder(tmp_path, cfg)
    p = M.tokens(cfg, 9)
    assert main(["generate", "--model", str(tmp_path), "--dtype", "float32", "--tokens", ",".join(map(str, p)), "--n", "6"]) == 0
    assert [int(x) for x in capsys.readouterr().out.split()] == M.greedy(cfg, w, p, 6)
    assert main(["generate", "--model", str(tmp_path), "--tokens", "1 2 3", "--n", "4", "--temperature", "0.8", "--top-k", "5"]) == 0
    assert len(capsys.readouterr().out.split()) == 4


def test_trace_through_the_runner(tmp_path):
    """bin/trace_run as a process of its own, both number formats."""
    import json
    import subprocess
    from pathlib import Path
    cfg = M.CONFIGS["tiny"]
    w = M.folder(tmp_path / "m", cfg)
    t = M.tokens(cfg, 12)
    ref = N.forward(cfg, w, t)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": t[:7], "want": [6, 2]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": t[7:8], "want": [0]}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": t[8:], "want": [3]}], "end": ["x"]}]
    for dt in ("bfloat16", "float32"):
        out = tmp_path / dt
        out.mkdir()
        r = subprocess.run([str(Path(__file__).resolve().parent.parent / "bin" / "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dt,
                            "--out", str(out), "--max-tokens", "12"], input="".join(json.dumps(s) + "\n" for s in steps), text=True,
                           capture_output=True, timeout=280)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [x for x in r.stdout.split("\n") if x.startswith("done")] == ["done 0", "done 1", "done 2"]
        got = np.concatenate([np.fromfile(out / ("%d.f32" % i), "<f4").reshape(-1, cfg["vocab"]) for i in range(3)])
        assert M.row_errors(got, ref[[6, 2, 7, 11]]).max() <= (1e-4 if dt == "float32" else 0.1)


def test_bad_calls_are_refused(ctx, tmp_path):
    import runit_mac_b200 as R
    s = Served(ctx, tmp_path, M.CONFIGS["tiny"], "bfloat16", max_seq=20)
    s.m.forward([1, 2, 3], 0)
    before = ctx.launches
    for call in (lambda: s.m.forward([1, 2], 5), lambda: s.m.forward([1] * 21, 0), lambda: s.m.forward([99, 1], 0),
                 lambda: s.m.forward([1, 2], 0, [2]), lambda: s.m.set_depth(7)):
        with pytest.raises(R.KernelError):
            call()
    assert ctx.launches == before


def test_buffers_are_aligned_whatever_was_allocated_before(ctx):
    """Odd small buffers first: the scratch of the batched blocks must still start at a multiple of 1024 bytes."""
    keep = [ctx.new_buffer(n) for n in (16, 700, 513, 1 << 12, 300, 90000, 256, 1100)]
    assert all(b.ptr % 1024 == 0 for b in keep)
    for b in keep[::2]:
        b.free()
    again = [ctx.new_buffer(n) for n in (512, 40, 5000)]
    a = np.arange(10, dtype=np.int32)
    assert all(b.ptr % 1024 == 0 for b in again) and (again[0].upload(a).download(np.int32, 10) == a).all()
