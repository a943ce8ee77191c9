"""GPU tests of the Pagazen decoder and the mechanisms it is made of, against the plain implementation (oracle/pagazen.py)."""
import ctypes as C
import json
import subprocess
from pathlib import Path

import numpy as np
import pytest

import pagazen_models as M
from oracle import pagazen as P
from oracle.nuvilorn import from_bf16, to_bf16

pytestmark = pytest.mark.gpu

EXACT = 3e-5         # row error (relative to the spread of the logits) in 32-bit


def bf16_rows(a):
    """bf16 bit patterns with rows padded to multiples of 8, and the values they hold."""
    a = np.asarray(a, np.float32)
    u = np.zeros(a.shape[:-1] + ((a.shape[-1] + 7) // 8 * 8,), np.uint16)
    u[..., :a.shape[-1]] = to_bf16(a).reshape(a.shape)
    return u, from_bf16(u)[..., :a.shape[-1]].astype(np.float64)


def close(got, ref, tol):
    """Within tol of the larger of the value itself and the root mean square."""
    got, ref = np.asarray(got, np.float64), np.asarray(ref, np.float64)
    assert np.isfinite(got).all()
    err = (np.abs(got - ref) / np.maximum(np.abs(ref), max(np.sqrt((ref ** 2).mean()), 1e-30))).max()
    assert err <= tol, err


class Rows:
    """Rows of values on the device in the operand type, and back."""

    def __init__(self, ctx, a, f32):
        a = np.asarray(a, np.float32)
        self.f32, self.shape, self.ld = f32, a.shape, (a.shape[1] + 7) // 8 * 8
        pad = np.zeros((a.shape[0], self.ld), np.float32)
        pad[:, :a.shape[1]] = a
        self.buf = ctx.buffer_from(pad if f32 else to_bf16(pad).reshape(pad.shape))
        self.values = (a if f32 else from_bf16(to_bf16(a)).reshape(a.shape)).astype(np.float64)

    def read(self):
        n = self.shape[0] * self.ld
        x = self.buf.download(np.float32, n) if self.f32 else from_bf16(self.buf.download(np.uint16, n))
        return x.reshape(self.shape[0], self.ld)[:, :self.shape[1]]

    def at(self, column):
        return self.buf.ptr + column * (4 if self.f32 else 2)


# ── norms, products with something in front ──
@pytest.mark.parametrize("T,width", [(1, 8), (3, 100), (5, 1003), (2, 2048)])
def test_add_norm_rows(ctx, T, width):
    import runit_mac_b200 as R
    g = np.random.default_rng(T)
    x, y = g.normal(size=(T, width)).astype(np.float32), (g.normal(size=(T, width)) * 10.0 ** -np.arange(T)[:, None]).astype(np.float32)
    gain, fin = g.uniform(0.5, 1.5, width).astype(np.float32), g.uniform(0.5, 1.5, width).astype(np.float32)
    gb, fb, ld = ctx.buffer_from(gain), ctx.buffer_from(fin), (width + 7) // 8 * 8
    ref = x + P.norm_offset(y.astype(np.float64), gain.astype(np.float64) - 1, 1e-3)
    for f32 in (1, 0):
        for final in (0, 1):
            xb, out = ctx.buffer_from(x), ctx.new_buffer(T * ld * 4)
            R.add_norm_rows(ctx, xb, ctx.buffer_from(y), gb, 1e-3, fb if final else None, out, f32, T, width)
            ctx.flush()
            got = (out.download(np.float32, T * ld) if f32 else from_bf16(out.download(np.uint16, T * ld))).reshape(T, ld)
            close(xb.download(np.float32, T * width).reshape(T, width), ref, 1e-5)
            close(got[:, :width], P.norm_offset(ref, fin.astype(np.float64) - 1, 1e-3) if final else ref, 1e-5 if f32 else 1e-2)
            assert (got[:, width:] == 0).all()


@pytest.mark.parametrize("m,k", [(1, 8), (7, 20), (65, 300), (200, 1001), (333, 1032), (9000, 640), (64, 2500), (40, 12000)])
def test_gemv_behind_a_residual_norm(ctx, m, k):
    import runit_mac_b200 as R
    g = np.random.default_rng(m)
    u, w = bf16_rows(g.normal(size=(m, k)) / np.sqrt(k))
    x, y = g.normal(size=k).astype(np.float32), g.normal(size=k).astype(np.float32)
    gy, gx = g.uniform(0.5, 1.5, k).astype(np.float32), g.uniform(0.5, 1.5, k).astype(np.float32)
    wb, xb, yb, gyb, gxb = (ctx.buffer_from(a) for a in (u, x, y, gy, gx))
    out, xo = ctx.new_buffer(m * 4), ctx.new_buffer(k * 4)
    new = x + P.norm_offset(y.astype(np.float64), gy.astype(np.float64) - 1, 1e-2)
    R.gemv_bf16_residual_f32(ctx, wb, xb, yb, gyb, None, xo, out, 1e-2, 0.0, 0, m, k)
    ctx.flush()
    close(out.download(np.float32, m), w @ new, 2e-5)
    close(xo.download(np.float32, k), new, 1e-5)
    R.gemv_bf16_residual_f32(ctx, wb, xb, yb, gyb, gxb, None, out, 1e-2, 1.5, 0, m, k)
    ctx.flush()
    z = w @ P.norm_offset(new, gx.astype(np.float64) - 1, 1e-2)
    close(out.download(np.float32, m), P.softcap(z, 1.5), 2e-5)
    R.gemv_bf16_residual_f32(ctx, wb, xb, None, None, gxb, None, out, 1e-2, 0.0, 1, m, k)
    ctx.flush()
    z = w @ P.norm_offset(x.astype(np.float64), gx.astype(np.float64) - 1, 1e-2)
    close(out.download(np.float32, m), np.maximum(z, 0) ** 2, 5e-5)


@pytest.mark.parametrize("plain,groups,group,m", [(0, 1, 24, 5), (13, 3, 7, 33), (64, 8, 32, 100), (0, 2, 640, 70), (24, 40, 48, 300), (0, 3, 4, 2), (128, 5, 96, 257)])
def test_gemv_behind_group_norms(ctx, plain, groups, group, m):
    import runit_mac_b200 as R
    k = plain + groups * group
    g = np.random.default_rng(m)
    u, w = bf16_rows(g.normal(size=(m, k)) / np.sqrt(k))
    x, f = g.normal(size=k).astype(np.float32), g.normal(size=k - plain).astype(np.float32)
    ref = w @ np.concatenate([x[:plain], (P.rms(x[plain:].astype(np.float64).reshape(groups, group), 1e-3).reshape(-1) * f)])
    wb, xb, fb, out = ctx.buffer_from(u), ctx.buffer_from(x), ctx.buffer_from(f), ctx.new_buffer(m * 4)
    R.gemv_bf16_groups_f32(ctx, wb, xb, fb, None, 0, out, 1e-3, plain, group, m, k)
    ctx.flush()
    close(out.download(np.float32, m), ref, 2e-5)
    parts = np.array([[(s ** 2).sum() for s in np.array_split(row, 3)] for row in x[plain:].reshape(groups, group)], np.float32)
    R.gemv_bf16_groups_f32(ctx, wb, xb, fb, ctx.buffer_from(parts), 3, out, 1e-3, plain, group, m, k)
    ctx.flush()
    close(out.download(np.float32, m), ref, 2e-5)


@pytest.mark.parametrize("n,group", [(24, 8), (35, 5), (512, 128), (4096, 4096), (3000, 1000), (8192, 64), (9000, 9000), (640, 320)])
@pytest.mark.parametrize("f32", [1, 0])
def test_gated_norm_rows(ctx, n, group, f32):
    import runit_mac_b200 as R
    T = 5
    g = np.random.default_rng(n)
    z = Rows(ctx, g.normal(size=(T, n)), f32)
    w = g.uniform(0.5, 1.5, n).astype(np.float32)
    src = g.normal(size=(T, n)) * 10.0 ** -np.arange(T)[:, None]
    for before in (1, 0):
        a = Rows(ctx, src, f32)
        R.gated_norm_rows(ctx, f32, a.buf, a.ld, n, group, z.buf, z.ld, before, ctx.buffer_from(w), 0.6, 1e-4, T)
        ctx.flush()
        v = a.values * P.silu(z.values) if before else a.values
        v = P.rms(v.reshape(T, -1, group), 1e-4).reshape(T, n)
        ref = v * w if before else v * P.silu(z.values) * 0.6
        got = a.read()
        for t in range(T):
            close(got[t], ref[t], 2e-5 if f32 else 2e-2)


# ── attention over a window ──
def _attn_case(ctx, H, G, d, dv, window, n, f32, seed, unit=1, slopes=True, cap=None):
    import runit_mac_b200 as R
    g = np.random.default_rng(seed)
    x = g.normal(size=(n, H * d + G * (d + dv)))
    proj = Rows(ctx, x, f32)
    cap = cap or n
    kd, vd = (d + 7) // 8 * 8, (dv + 7) // 8 * 8
    kc, vc = ctx.buffer_from(np.zeros(G * cap * kd, np.float32)), ctx.buffer_from(np.zeros(G * cap * vd, np.float32))
    sl = P.head_slopes(H) if slopes else np.zeros(H)
    sb = ctx.buffer_from(sl.astype(np.float32))
    scale = 4 * d ** -0.5                                           # sharp: single keys count
    cfg = R.HeadsCfg(H, G, d, dv, window, cap, unit, scale, 0.7, 1e-5, sb.ptr if slopes else None, kc.ptr, vc.ptr)
    v = proj.values
    q, k, vv = v[:, :H * d].reshape(n, H, d), v[:, H * d:H * d + G * d].reshape(n, G, d), v[:, H * d + G * d:].reshape(n, G, dv)
    if unit:
        q, k = P.rms(q, 1e-5), P.rms(k, 1e-5)
    own = np.arange(H) // (H // G)
    p = P.softmax_visible(P.biased_scores(q, k[:, own], scale, sl), P.window_mask(n, window or n))
    ref = 0.7 * np.einsum("hij,jhd->ihd", p, vv[:, own]).reshape(n, H * dv)
    return cfg, proj, ref, (kc, vc, sb)


ATTN = [(4, 2, 48, 40, 20, 70, 0), (8, 1, 128, 128, 100, 200, 60), (20, 2, 64, 64, 0, 130, 3), (3, 3, 7, 5, 1, 40, 8), (2, 1, 192, 160, 64, 150, 1),
        (12, 4, 33, 70, 65, 129, 64), (5, 1, 16, 24, 1000, 90, 30), (2, 2, 256, 264, 30, 50, 20)]


@pytest.mark.parametrize("case", range(len(ATTN)))
@pytest.mark.parametrize("f32", [1, 0])
@pytest.mark.parametrize("unit,slopes", [(1, True), (0, False)])
def test_attention_rows(ctx, case, f32, unit, slopes):
    """Whole, and in portions that start anywhere, in a cache that holds everything and in one that wraps around."""
    import runit_mac_b200 as R
    H, G, d, dv, window, n, start = ATTN[case]
    for cap in ({n, window - 1 + n - start} if window else {n}):
        cfg, proj, ref, keep = _attn_case(ctx, H, G, d, dv, window, n, f32, case, unit, slopes, max(cap, 1))
        out = Rows(ctx, np.zeros((n, H * dv)), f32)
        part, tick = ctx.new_buffer(1 << 20), ctx.buffer_from(np.zeros(4096, np.uint32))
        es = 4 if f32 else 2
        for a, b in ((0, start), (start, n)):
            at = a
            while at < b:
                T = min(b - at, n if cap >= n else cap - window + 1)
                R.heads_rows(ctx, C.byref(cfg), None, f32, proj.buf.ptr + at * proj.ld * es, proj.ld, T, at)
                R.head_attention_rows(ctx, C.byref(cfg), f32, proj.buf.ptr + at * proj.ld * es, proj.ld, out.buf.ptr + at * out.ld * es, out.ld, T, at,
                                      part, (1 << 20) // 4, tick)
                at += T
        ctx.flush()
        close(out.read(), ref, 3e-5 if f32 else 5e-2)


@pytest.mark.parametrize("case", range(len(ATTN)))
@pytest.mark.parametrize("f32", [1, 0])
@pytest.mark.parametrize("nsplit", [1, 3, 16, 64])
def test_attention_step(ctx, case, f32, nsplit):
    import runit_mac_b200 as R
    H, G, d, dv, window, n, _ = ATTN[case]
    cfg, proj, ref, keep = _attn_case(ctx, H, G, d, dv, window, n, 1, case)
    ref_rows = {}
    rows = proj.read().astype(np.float32)
    part, tick = ctx.new_buffer(H * 64 * (dv + 2) * 4), ctx.buffer_from(np.zeros(4096, np.uint32))
    ao, dummy = ctx.new_buffer(H * dv * 4), ctx.new_buffer(16)
    for t in range(n):
        if t < n - 4:            # earlier positions: their cache rows only
            if t == 0:
                Rb = Rows(ctx, rows[:n - 4], f32)
                R.heads_rows(ctx, C.byref(cfg), None, f32, Rb.buf, Rb.ld, n - 4, 0)
                ctx.flush()
            continue
        pb = ctx.buffer_from(np.array([t], np.int32))
        R.heads_step(ctx, C.byref(cfg), None, f32, ctx.buffer_from(rows[t]), ao, dummy, dummy, part, tick, nsplit, pb)
        ctx.flush()
        ref_rows[t] = ao.download(np.float32, H * dv)
        assert (tick.download(np.uint32, 4096) == 0).all()
    for t, got in ref_rows.items():
        close(got, ref[t], 3e-5 if f32 else 5e-2)


# ── recurrences ──
LINEAR = [(2, 2, 32, 48), (4, 1, 64, 64), (6, 3, 40, 16), (2, 1, 128, 130), (2, 2, 256, 100), (3, 1, 5, 7), (2, 2, 300, 33), (4, 2, 16, 32)]


@pytest.mark.parametrize("case", range(len(LINEAR)))
@pytest.mark.parametrize("f32", [1, 0])
@pytest.mark.parametrize("with_dt", [0, 1])
def test_linear_rows(ctx, case, f32, with_dt):
    """One pass, and portions that carry the state on (a step, 15 tokens, chunk edges)."""
    import runit_mac_b200 as R
    H, G, dk, dv = LINEAR[case]
    n = 300
    g = np.random.default_rng(case)
    q, k, v = Rows(ctx, g.normal(size=(n, G * dk)), f32), Rows(ctx, g.normal(size=(n, G * dk)) / np.sqrt(dk), f32), Rows(ctx, g.normal(size=(n, H * dv)), f32)
    decay = np.array([1 - 2.0 ** -(1 + 2 * h) for h in range(H)], np.float32)
    decay[0] = 1.0 if case % 2 else 0.02
    ld = np.log(decay)
    dt = g.uniform(0.01, 2.0, (n, H)).astype(np.float32)
    skip = g.normal(size=H).astype(np.float32)
    own = np.arange(H) // (H // G)
    kk = k.values.reshape(n, G, dk)[:, own]
    a = np.broadcast_to(decay.astype(np.float64), (n, H))
    if with_dt:
        kk, a = kk * dt[..., None], np.exp(ld * dt.astype(np.float64))
    vv = v.values.reshape(n, H, dv)
    ref = P.linear_scan(q.values.reshape(n, G, dk)[:, own], kk, vv, a)
    if with_dt:
        ref = ref + skip[:, None] * vv
    ref = ref.reshape(n, H * dv)
    es = 4 if f32 else 2
    db, lb, sb, tb = ctx.buffer_from(decay), ctx.buffer_from(ld), ctx.buffer_from(skip), ctx.buffer_from(dt)
    nbytes = ctx.lib.runit_linear_scratch_bytes(H, dk, dv, n)
    scr = ctx.new_buffer(max(nbytes, 16))
    state = ctx.buffer_from(np.full(H * dk * dv, 7.0, np.float32))            # what an earlier sequence has left
    for cuts in ([n], [1, 15, 16, 127, 129, 12], [128, 172], [2, 298]):
        out, at = Rows(ctx, np.zeros((n, H * dv)), f32), 0
        for T in cuts:
            off = lambda r: r.buf.ptr + at * r.ld * es
            cfg = R.LinearCfg(H, G, dk, dv, q.ld, k.ld, v.ld, out.ld, off(q), off(k), off(v), tb.ptr + at * H * 4 if with_dt else None, lb.ptr, db.ptr,
                              sb.ptr if with_dt else None, state.ptr, off(out))
            R.linear_rows(ctx, C.byref(cfg), f32, scr if nbytes else None, T, at)
            at += T
        ctx.flush()
        close(out.read(), ref, 5e-5 if f32 else 4e-2)


@pytest.mark.parametrize("H,G,dv,N,taps", [(4, 1, 24, 16, 4), (6, 3, 16, 40, 5), (3, 1, 5, 7, 2), (2, 2, 64, 128, 4), (1, 1, 1, 1, 1), (2, 1, 40, 280, 7)])
def test_state_space_step_and_convolution(ctx, H, G, dv, N, taps):
    """Token by token, and the convolution of portions that leave their last inputs behind."""
    import runit_mac_b200 as R
    n, inner = 40, H * dv
    ch = inner + 2 * G * N
    g = np.random.default_rng(H * N)
    raw = g.normal(size=(n, inner + ch + H)).astype(np.float32)
    w, b = g.normal(0, 0.5, (ch, taps)).astype(np.float32), g.normal(0, 0.2, ch).astype(np.float32)
    bias, a, skip = g.uniform(-3, 0, H).astype(np.float32), -g.uniform(0.2, 3, H).astype(np.float32), g.normal(size=H).astype(np.float32)
    f8 = lambda x: x.astype(np.float64)
    conv = P.silu(P.causal_conv(f8(raw[:, inner:inner + ch]), f8(w), f8(b)))
    dt = P.softplus(f8(raw[:, inner + ch:]) + bias)
    own = np.arange(H) // (H // G)
    x, B, Cc = conv[:, :inner].reshape(n, H, dv), conv[:, inner:inner + G * N].reshape(n, G, N)[:, own], conv[:, inner + G * N:].reshape(n, G, N)[:, own]
    y = P.linear_scan(Cc, B * dt[..., None], x, np.exp(f8(a) * dt)) + skip[:, None] * x
    ref = y.reshape(n, inner) * P.silu(f8(raw[:, :inner]))
    bufs = [ctx.buffer_from(t) for t in (w, b, bias, a, skip)]
    state, ring = ctx.buffer_from(np.full(H * N * dv, 9.0, np.float32)), ctx.buffer_from(np.full(taps * ch, 9.0, np.float32))
    cfg = R.SsmCfg(H, dv, N, G, taps, *(t.ptr for t in bufs), state.ptr, ring.ptr)
    ns = (dv + 31) // 32
    yb, sq = ctx.new_buffer(inner * 4), ctx.new_buffer(H * ns * 4)
    for t in range(n):
        R.ssm_step(ctx, C.byref(cfg), ctx.buffer_from(raw[t]), yb, sq, ctx.buffer_from(np.array([t], np.int32)))
        ctx.flush()
        got = yb.download(np.float32, inner)
        close(got, ref[t], 5e-5)
        close(sq.download(np.float32, H * ns).sum(), (ref[t] ** 2).sum(), 2e-4)
    for f32 in (1, 0):
        for cuts in ([n], [1, 2, 3, 34], [33, 7]):
            at, outs = 0, []
            for T in cuts:
                pr, xbc = Rows(ctx, raw[at:at + T, :inner + ch], f32), Rows(ctx, np.zeros((T, ch)), f32)
                db = ctx.buffer_from(raw[at:at + T, inner + ch:])
                R.ssm_conv_rows(ctx, C.byref(cfg), f32, pr.buf, pr.ld, xbc.buf, xbc.ld, db, T, at)
                ctx.flush()
                outs.append(xbc.read())
                close(db.download(np.float32, T * H).reshape(T, H), dt[at:at + T], 1e-5)
                at += T
            close(np.concatenate(outs), conv, 1e-5 if f32 else 3e-2)


@pytest.mark.parametrize("H,d,dv,rot", [(2, 32, 48, 32), (3, 10, 7, 6), (1, 256, 160, 100), (2, 130, 33, 0)])
def test_retention_step(ctx, H, d, dv, rot):
    import runit_mac_b200 as R
    n, g = 30, np.random.default_rng(d)
    raw = g.normal(size=(n, 2 * H * (d + dv))).astype(np.float32)
    decay = np.array([0.5, 0.9, 1.0][:H], np.float32)
    v8 = raw.astype(np.float64)
    q, k = P.rotate_halves(v8[:, :H * d].reshape(n, H, d), np.arange(n), rot, 50.0), P.rotate_halves(v8[:, H * d:2 * H * d].reshape(n, H, d), np.arange(n), rot, 50.0)
    ref = P.linear_scan(q, k * d ** -0.5, v8[:, 2 * H * d:2 * H * d + H * dv].reshape(n, H, dv), np.broadcast_to(decay.astype(np.float64), (n, H)))
    f = 50.0 ** (-2.0 * np.arange(max(rot // 2, 1)) / max(rot, 1))
    freq, db = ctx.buffer_from(np.stack([np.float32(f), np.float32(f - np.float32(f))])), ctx.buffer_from(np.stack([decay, np.log(decay)]))
    state = ctx.buffer_from(np.full(H * d * dv, 3.0, np.float32))
    cfg = R.RetentionCfg(H, d, dv, rot, 0.6, freq.ptr, db.ptr, state.ptr)
    ao, fac, sq = ctx.new_buffer(H * dv * 4), ctx.new_buffer(H * dv * 4), ctx.new_buffer(H * ((dv + 31) // 32) * 4)
    for t in range(n):
        R.heads_step(ctx, None, C.byref(cfg), 1, ctx.buffer_from(raw[t]), ao, fac, sq, None, None, 1, ctx.buffer_from(np.array([t], np.int32)))
        ctx.flush()
        close(ao.download(np.float32, H * dv), ref[t].reshape(-1), 5e-5)
        close(sq.download(np.float32, H * ((dv + 31) // 32)).reshape(H, -1).sum(1), (ref[t] ** 2).sum(1), 2e-4)
        close(fac.download(np.float32, H * dv), 0.6 * P.silu(v8[t, 2 * H * d + H * dv:]), 1e-5)


@pytest.mark.parametrize("rot,base", [(64, 10000.0), (20, 50.0)])
def test_rotation_at_far_positions(ctx, rot, base):
    """Angles of thousands of radians keep the precision of their sine and cosine."""
    import runit_mac_b200 as R
    g, n, start = np.random.default_rng(rot), 16, 30000
    raw = g.normal(size=(n, 4 * rot)).astype(np.float32)
    f = base ** (-2.0 * np.arange(rot // 2) / rot)
    freq, db, state = ctx.buffer_from(np.stack([np.float32(f), np.float32(f - np.float32(f))])), ctx.buffer_from(np.zeros(2, np.float32)), ctx.new_buffer(rot * rot * 4)
    cfg = R.RetentionCfg(1, rot, rot, rot, 1.0, freq.ptr, db.ptr, state.ptr)
    pr = Rows(ctx, raw, 1)
    R.heads_rows(ctx, None, C.byref(cfg), 1, pr.buf, pr.ld, n, start)
    ctx.flush()
    ref = P.rotate_halves(raw[:, None, :rot].astype(np.float64), start + np.arange(n), rot, base)[:, 0]
    assert np.abs(pr.read()[:, :rot] - ref).max() <= 2e-6


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


def check_rows(got, ref, dtype):
    e = M.row_errors(got, ref)
    if dtype == "float32":
        assert e.max() <= EXACT, e.max()
    else:
        assert np.median(e) <= 0.03 and (e > 0.1).mean() <= 0.02, (np.median(e), np.sort(e)[-5:])


@pytest.mark.parametrize("name", sorted(M.CONFIGS))
@pytest.mark.parametrize("n", [1, 2, 15, 16, 150])
def test_prompt(ctx, tmp_path, dtype, name, n):
    s = Served(ctx, tmp_path, M.CONFIGS[name], dtype)
    t = M.tokens(s.cfg, n)
    check_rows(s.run(t, [n]), P.forward(s.cfg, s.w, t), dtype)


@pytest.mark.parametrize("name", sorted(M.CONFIGS))
def test_prefill_against_token_by_token_and_portions(ctx, tmp_path, dtype, name):
    s = Served(ctx, tmp_path, M.CONFIGS[name], dtype)
    t = M.tokens(s.cfg, 140)
    ref = P.forward(s.cfg, s.w, t)
    whole = s.run(t, [140])
    for cuts in ([1], [2], [3, 2], [31, 1, 33], [128, 12], [139, 1], [7, 50, 2], [17]):
        check_rows(s.run(t, cuts), ref, dtype)
    if dtype == "float32":
        assert M.row_errors(s.run(t, [1]), whole).max() <= EXACT


def test_layer_by_layer(ctx, tmp_path):
    s = Served(ctx, tmp_path, M.CONFIGS["mixed"], "float32")
    t = M.tokens(s.cfg, 45)
    _, trail = P.forward(s.cfg, s.w, t, want_layers=True)
    s.m.set_depth(0)
    s.m.forward(t, 0)
    close(s.m.residual(45), np.asarray(s.w["embed"], np.float64)[t] * s.cfg["embedding"]["scale"], 1e-6)
    for d in range(1, len(trail) + 1):
        s.m.set_depth(d)
        s.m.forward(t, 0)
        close(s.m.residual(45), trail[d - 1], 5e-5)


ALONE = {
    "window attention": ([(M.parallel(M.left(6, 2, 24, 40, 11), M.right(1, 8, 8, 8)), None)], ["l0.mix.right.o"]),
    "a window of one": ([(M.parallel(M.left(2, 1, 16, 16, 1), M.right(1, 8, 8, 8)), None)], ["l0.mix.right.o"]),
    "as many key heads": ([(M.parallel(M.left(3, 3, 24, 8, 50), M.right(1, 8, 8, 8)), None)], ["l0.mix.right.o"]),
    "retention": ([(M.parallel(M.left(1, 1, 8, 8, 4), M.right(3, 40, 24, 40)), None)], ["l0.mix.left.o"]),
    "retention, some dimensions rotated": ([(M.parallel(M.left(1, 1, 8, 8, 4), M.right(2, 24, 72, 10, base=30.0)), None)], ["l0.mix.left.o"]),
    "retention, one head that keeps everything": ([(M.parallel(M.left(1, 1, 8, 8, 4), M.right(1, 16, 16, 16, decay=[1.0])), None)], ["l0.mix.left.o"]),
    "state space": ([(M.mamba(4, 16, 24), None)], []),
    "state space, groups": ([(M.mamba(6, 8, 16, groups=2, norm_groups=3), None)], []),
    "state space, norm groups inside heads": ([(M.mamba(2, 24, 16, conv=3, norm_groups=6), None)], []),
    "state space, one tap": ([(M.mamba(2, 24, 16, conv=1), None)], []),
    "feed-forward": ([(M.mamba(1, 8, 8), 40)], ["l0.mix.o"]),
    "tensors used twice": ([(M.mamba(2, 16, 16), 24), 0, (M.parallel(M.left(2, 1, 16, 16, 6), M.right(2, 16, 16, 16)), 24), 2, 0], []),
}


@pytest.mark.parametrize("name", sorted(ALONE))
def test_mechanism_alone(ctx, tmp_path, dtype, name):
    """One mechanism per model; the output projection of what is not looked at is zero."""
    layers, zero = ALONE[name]
    cfg = M.config(48, 60, layers)

    def edit(w):
        for z in zero:
            w[z][:] = 0
    s = Served(ctx, tmp_path, cfg, dtype, edit=edit)
    t = M.tokens(cfg, 140)
    ref = P.forward(cfg, s.w, t)
    for cuts in ([140], [1], [20, 3], [90, 2, 48]):
        check_rows(s.run(t, cuts), ref, dtype)


def _swap(name, make):
    return lambda mp: mp.setattr(P, name, make(getattr(P, name)))


def _window(f, n, size, by):
    return f(n, max(size + by, 1))


def _neighbours(x, pos, dims, base):
    out, a = np.array(x), np.asarray(pos)[:, None] * float(base) ** (-2.0 * np.arange(dims // 2) / dims)
    c, s = np.cos(a)[:, None], np.sin(a)[:, None]
    out[..., 0:dims:2], out[..., 1:dims:2] = x[..., 0:dims:2] * c - x[..., 1:dims:2] * s, x[..., 1:dims:2] * c + x[..., 0:dims:2] * s
    return out


def _first_dropped(q, k, v, a):
    """The state forgets what came before position 40."""
    out = P.linear_scan_kept(q, k, v, a)
    out[40:] = P.linear_scan_kept(q[40:], k[40:], v[40:], a[40:])
    return out


FAULTS = {
    "a window one longer": _swap("window_mask", lambda f: lambda n, z: _window(f, n, z, 1)),
    "a window one shorter": _swap("window_mask", lambda f: lambda n, z: _window(f, n, z, -1)),
    "no distance bias": _swap("head_slopes", lambda f: lambda h: 0.0 * f(h)),
    "slopes in reverse": _swap("head_slopes", lambda f: lambda h: f(h)[::-1]),
    "neighbours rotated instead of halves": _swap("rotate_halves", lambda f: _neighbours),
    "no rotation": _swap("rotate_halves", lambda f: lambda x, p, d, b: x),
    "a state that is lost": _swap("linear_scan", lambda f: _first_dropped),
    "decay after the key": _swap("linear_scan", lambda f: lambda q, k, v, a: f(q, k * a[..., None], v, a)),
    "the next token's tap": _swap("causal_conv", lambda f: lambda x, w, b: f(x, w[:, ::-1], b)),
    "a convolution without history": _swap("causal_conv", lambda f: lambda x, w, b: np.concatenate([f(x[:40], w, b), f(x[40:], w, b)])),
    "no softplus": _swap("softplus", lambda f: lambda z: np.maximum(z, 0)),
    "no cap": _swap("softcap", lambda f: lambda z, c: z),
    "norm weights not around one": _swap("norm_offset", lambda f: lambda x, w, e: f(x, w - 1, e) + 1e-3),
    "the feed-forward's square": _swap("relu2_ff", lambda f: lambda h, u, d: np.maximum(h @ u.T, 0) @ d.T),
}


def test_faults_would_show(ctx, tmp_path):
    """A mistake in the plain implementation moves its logits far beyond the tolerances above, away from what the decoder
    computes in prompts, in portions and in decoding."""
    cfg = M.config(96, 131, [(M.parallel(M.left(4, 2, 32, 32, 12, scale=0.6), M.right(3, 24, 24, 24, base=100.0)), 64), (M.mamba(4, 16, 16, groups=2), 64), 0, 1])
    s = Served(ctx, tmp_path, cfg, "float32")
    t = M.tokens(cfg, 80)
    runs = [s.run(t, [80]), s.run(t, [40] + [1] * 40), s.run(t, [9, 2])]
    ref = P.forward(cfg, s.w, t)
    assert max(M.row_errors(r, ref).max() for r in runs) <= EXACT
    P.linear_scan_kept = P.linear_scan
    for what, plant in FAULTS.items():
        with pytest.MonkeyPatch.context() as mp:
            plant(mp)
            bad = P.forward(cfg, s.w, t)
        for got in runs:
            e = M.row_errors(got, bad)
            assert e[40:].max() > 0.01, (what, e[40:].max())
    del P.linear_scan_kept


@pytest.mark.parametrize("window", [1, 2, 63, 64, 65, 100, 128])
def test_keys_at_the_edge_of_the_window(ctx, tmp_path, dtype, window):
    """One token has a key of its own that an asking token looks for: just inside the window it takes nearly all the weight, one
    position further it does not exist; in prompts, at every cut and in decoding."""
    cfg = M.config(64, 40, [(M.parallel(M.left(1, 1, 32, 32, window, scale=1.5), M.right(1, 8, 8, 8)), None)], scale=1.0)
    MARK, ASK = 38, 39

    def edit(w):
        w["l0.mix.right.o"][:] = 0
        w["embed"][:] = np.random.default_rng(3).normal(size=w["embed"].shape)
        w["embed"][:, :2] = 0
        w["embed"][MARK, 0], w["embed"][ASK, 1] = 12.0, 12.0
        key = np.ones(32)
        key[::2] = -1                                              # the mark's key and the asking query are the same vector
        w["l0.mix.left.k"][:, 0], w["l0.mix.left.q"][:, 1] = key, key
    s = Served(ctx, tmp_path, cfg, dtype, edit=edit)
    for back, inside in ((window - 1, True), (window, False)):
        for at in (window + 3, 140, 200):
            t = [int(x) for x in np.random.default_rng(at).integers(0, 38, at + 1)]
            t[at] = ASK
            plain = P.forward(cfg, s.w, t)[at:]
            if back:
                t[at - back] = MARK
            ref = P.forward(cfg, s.w, t)[at:]
            moved = M.row_errors(plain, ref).max()
            if back:
                assert (moved > 0.2) if inside else (moved < 1e-9), moved
            for cuts in ([at + 1], [at, 1], [max(at - 5, 1), 6], [50], [max(at - back, 1), 1]):
                got = s.run(t, cuts, want=[at])
                assert M.row_errors(got, ref).max() <= (1e-4 if dtype == "float32" else 0.06)


@pytest.mark.parametrize("far", [0, 1, 127, 128, 129, 200])
def test_one_token_far_back_in_the_state(ctx, tmp_path, dtype, far):
    """A head that forgets nothing, a token whose value alone is not zero and a query that asks for its key: the answer hangs on
    one token at a chunk's edge, at the start or hundreds of tokens back."""
    cfg = M.config(64, 40, [(M.parallel(M.left(1, 1, 8, 8, 2), M.right(1, 32, 32, 32, base=1e6, decay=[1.0])), None)], scale=1.0)
    MARK, ASK = 38, 39

    def edit(w):
        w["l0.mix.left.o"][:] = 0
        w["embed"][:, :2] = 0
        w["embed"][MARK, 0] = 20.0
        w["embed"][ASK, 1] = 20.0
        for n in "kv":
            w["l0.mix.right." + n][:] *= 0.05
            w["l0.mix.right." + n][:, 0] = np.random.default_rng(1).normal(size=32)
            w["l0.mix.right." + n][:, 1] = 0
        w["l0.mix.right.q"][:, 1] = w["l0.mix.right.k"][:, 0]
    s = Served(ctx, tmp_path, cfg, dtype, edit=edit)
    t = [int(x) for x in np.random.default_rng(far).integers(0, 38, 300)]
    t[far] = MARK
    t[290] = t[299] = ASK
    ref = P.forward(cfg, s.w, t)[[290, 299]]
    t2 = list(t)
    t2[far] = 7
    assert M.row_errors(P.forward(cfg, s.w, t2)[[290, 299]], ref).min() > 0.3
    for cuts in ([300], [280, 20], [128, 127, 5], [200] + [1] * 100, [2]):
        assert M.row_errors(s.run(t, cuts, want=[290, 299]), ref).max() <= (1e-4 if dtype == "float32" else 0.06)


def test_state_and_cache_are_used_again(ctx, tmp_path, dtype):
    """Sequences one after the other, longer and shorter, start from nothing whatever the last one has left."""
    s = Served(ctx, tmp_path, M.CONFIGS["mixed"], dtype)
    seqs = [M.tokens(s.cfg, n, n) for n in (150, 3, 60, 1, 17, 150)]
    refs = [P.forward(s.cfg, s.w, t) for t in seqs]
    for cuts in ([200], [1], [20, 1, 2]):
        for t, ref in zip(seqs, refs):
            check_rows(s.run(t, cuts), ref, dtype)


def test_portions_do_not_depend_on_what_ran_before(ctx, tmp_path, dtype):
    s = Served(ctx, tmp_path, M.CONFIGS["mixed"], dtype)
    a, b = M.tokens(s.cfg, 90, 1), M.tokens(s.cfg, 140, 2)
    first = s.run(a, [40, 50])
    s.run(b, [140])
    s.m.generate(b[:20], 30)
    assert (s.run(a, [40, 50]) == first).all()


def test_long_prompt_is_cut_inside(ctx, tmp_path, dtype):
    """Prompts longer than one batched portion (256 tokens in 32-bit, 2048 in bf16): the ring of a window wraps around."""
    cfg = M.config(32, 60, [(M.parallel(M.left(2, 1, 16, 16, 70), M.right(2, 16, 16, 8)), 32), (M.mamba(2, 16, 16), 32)])
    n = 600 if dtype == "float32" else 2300
    s = Served(ctx, tmp_path, cfg, dtype, max_seq=n + 200)
    t = M.tokens(cfg, n)
    want = [0, 255, 256, 257, 511, 512, n - 1] if dtype == "float32" else [0, 127, 128, 2047, 2048, 2049, 2117, 2118, n - 1]
    ref = P.forward(cfg, s.w, t)
    got = s.run(t, [n], want=want)
    assert M.row_errors(got, ref[want]).max() <= (1e-4 if dtype == "float32" else 0.1)
    nxt = s.m.prefill(t)
    top = np.sort(ref[-1])[-2:]
    assert nxt == int(np.argmax(ref[-1])) or (dtype == "bfloat16" and top[1] - top[0] < 0.1 * np.std(ref[-1]))


def test_long_decoding(ctx, tmp_path, dtype):
    """Decoded far past the window's ring (97 + 255 positions in 32-bit)."""
    cfg = M.config(48, 60, [(M.parallel(M.left(2, 1, 16, 16, 98), M.right(2, 16, 16, 8)), 32), (M.mamba(2, 16, 16), 32), 0])
    s = Served(ctx, tmp_path, cfg, dtype, max_seq=700)
    p = M.tokens(cfg, 3)
    out = s.m.generate_greedy(p, 640)[len(p) - 1:].tolist()
    seq = p + out
    ref = P.forward(cfg, s.w, seq[:-1])[len(p) - 1:]
    margin = ref.max(1) - ref[np.arange(len(out)), out]
    agree = (margin <= (1e-3 if dtype == "float32" else 0.25) * np.std(ref)).mean()
    assert agree == 1.0 if dtype == "float32" else agree > 0.95, agree
    rows = s.run(seq, [300] + [1] * 343, want=range(300, 643, 7))
    check_rows(rows, P.forward(cfg, s.w, seq)[300:643:7], dtype)


def test_wanted_places_keep_their_order(ctx, tmp_path):
    s = Served(ctx, tmp_path, M.CONFIGS["mixed"], "float32")
    t = M.tokens(s.cfg, 90)
    ref = P.forward(s.cfg, s.w, t)
    want = [89, 3, 3, 40] + list(range(80, 0, -1))
    assert M.row_errors(s.m.forward(t, 0, want), ref[want]).max() <= EXACT


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_greedy_generation(ctx, tmp_path, name):
    """Prefill and recorded decode steps, and the token-by-token path, give the plain implementation's continuation."""
    s = Served(ctx, tmp_path, M.CONFIGS[name], "float32")
    p = M.tokens(s.cfg, 21)
    ref = M.greedy(s.cfg, s.w, p, 40)
    assert len(set(ref)) > 3
    assert s.m.generate(p, 40).tolist() == ref
    assert s.m.generate_greedy(p, 39)[len(p) - 1:].tolist() == ref
    assert s.m.prefill(p) == ref[0]
    # steps and portions continue from where the last pass ended
    seq, got = list(p), [ref[0]]
    for _ in range(5):
        got.append(s.m.forward_greedy(got[-1], len(seq)))
        seq.append(got[-2])
    assert got == ref[:6]
    lg = s.m.forward(ref[5:9], len(p) + 5, [3])
    assert int(np.argmax(lg[0])) == ref[9]


def test_sampled_generation(ctx, tmp_path):
    import runit_mac_b200 as R
    s = Served(ctx, tmp_path, M.CONFIGS["mixed"], "bfloat16")
    p = M.tokens(s.cfg, 12)
    a, b, c = (s.m.generate_sampled(p, 30, R.SamplerCfg(0.9, 20, 0.95, 1.1, 0), seed=x) for x in (3, 3, 4))
    assert (a == b).all() and (a != c).any() and ((a[11:] >= 0) & (a[11:] < s.cfg["vocab"])).all()
    zero = s.m.generate_sampled(p, 30, R.SamplerCfg(0.0, 0, 1.0, 1.0, 0), seed=1)
    assert (zero[11:] == s.m.generate_greedy(p, 30)[11:]).all()


def test_a_pass_starts_at_zero_or_where_the_last_one_ended(ctx, tmp_path):
    import runit_mac_b200 as R
    s = Served(ctx, tmp_path, M.CONFIGS["tiny"], "bfloat16", max_seq=20)
    s.m.forward([1, 2, 3, 4], 0)
    for call in (lambda: s.m.forward([1, 2], 2), lambda: s.m.forward([1], 3), lambda: s.m.forward([1, 2], 5), lambda: s.m.forward_greedy(1, 2),
                 lambda: s.m.generate_greedy([1], 3, 2), lambda: s.m.forward([1] * 21, 0)):
        with pytest.raises(R.KernelError):
            call()
    s.m.forward([1, 2], 4)
    s.m.forward_greedy(1, 6)
    s.m.forward([1, 2], 0)


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
    """bin/trace_run as a process of its own, both number formats, two sequences."""
    cfg = M.CONFIGS["tiny"]
    w = M.folder(tmp_path / "m", cfg)
    t, u = M.tokens(cfg, 12), M.tokens(cfg, 5, 9)
    rt, ru = P.forward(cfg, w, t), P.forward(cfg, w, u)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": t[:7], "want": [6, 2]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": t[7:8], "want": [0]}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": t[8:], "want": [3]}], "end": ["x"]},
             {"step": 3, "entries": [{"id": "y", "tokens": u, "want": [4]}], "end": ["y"]}]
    for dt in ("bfloat16", "float32"):
        out = tmp_path / dt
        out.mkdir()
        r = subprocess.run([str(Path(__file__).resolve().parent.parent / "bin" / "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dt,
                            "--out", str(out), "--max-tokens", "12"], input="".join(json.dumps(s) + "\n" for s in steps), text=True,
                           capture_output=True, timeout=280)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [x for x in r.stdout.split("\n") if x.startswith("done")] == ["done %d" % i for i in range(4)]
        got = np.concatenate([np.fromfile(out / ("%d.f32" % i), "<f4").reshape(-1, cfg["vocab"]) for i in range(4)])
        assert M.row_errors(got, np.concatenate([rt[[6, 2, 7, 11]], ru[[4]]])).max() <= (1e-4 if dt == "float32" else 0.1)


# ── the same parts in other designs ──
class _Tensors:
    """A source of tensors from a dict, the values as bf16 holds them."""

    def __init__(self, w):
        self.w = {k: from_bf16(to_bf16(np.asarray(v))).reshape(np.shape(v)) for k, v in w.items()}

    def shape(self, n):
        return self.w[n].shape

    def f32(self, n):
        return self.w[n].astype(np.float32)

    def bf16(self, n):
        return to_bf16(self.w[n]).reshape(self.w[n].shape)


def _serve(ctx, R, up, layers, w, V, W, exact, post):
    head = {"embed": up.matrix([("embed", V)], W), "final_norm": up.values(w["final"]), "head": up.matrix([("head", V)], W)}
    cfg = R.LayeredCfg(n_layers=len(layers), width=W, vocab=V, max_seq=200, exact=exact, post_norm=post, eps=1e-5, embed_scale=2.0, logit_cap=9.0)
    return R.LayeredModel(ctx, cfg, layers, head, keep=up)


def _check_served(m, t, ref, exact):
    for cuts in ([len(t)], [1], [20, 3], [70, 30]):
        out, pos, i = [], 0, 0
        while pos < len(t):
            c = min(cuts[i % len(cuts)], len(t) - pos)
            out.append(m.forward(t[pos:pos + c], pos, range(c)))
            pos, i = pos + c, i + 1
        check_rows(np.concatenate(out), ref, "float32" if exact else "bfloat16")
    nxt = m.generate(t, 2)
    assert exact == 0 or int(nxt[0]) == int(np.argmax(ref[-1]))


@pytest.mark.parametrize("exact", [1, 0])
def test_mixers_behind_norms_with_one_gain(ctx, exact):
    """Attention alone (no window, no bias, queries and keys as they are), retention alone and a state-space layer, each behind
    a norm with one gain."""
    import runit_mac_b200 as R
    from runit_mac_b200 import models
    W, V, g = 56, 70, np.random.default_rng(2)
    lin = lambda r, c: g.normal(0, 1.2 / np.sqrt(c), (r, c))
    at, rt = M.left(4, 2, 16, 24, 10 ** 6), M.right(3, 16, 16, 8)
    ss = M.mamba(4, 16, 24, groups=2, norm_groups=2)["mixer"]
    inner, ch = 64, 64 + 96
    w = {"embed": lin(V, W) * 4, "head": lin(V, W) * 3, "final": np.array([1.2])}
    w.update({"a.q": lin(64, W), "a.k": lin(32, W), "a.v": lin(48, W), "a.o": lin(W, 96), "r.q": lin(48, W), "r.k": lin(48, W), "r.v": lin(48, W), "r.g": lin(48, W),
              "r.o": lin(W, 48), "s.in": lin(inner + ch + 4, W), "s.conv": g.normal(0, 0.5, (ch, 4)), "s.conv.b": g.normal(0, 0.2, ch), "s.dt_bias": g.uniform(-3, 0, 4),
              "s.A_log": g.uniform(-1, 1, 4), "s.D": g.normal(size=4), "s.norm": g.uniform(0.5, 1.5, inner), "s.o": lin(W, inner), "up": lin(40, W), "down": lin(W, 40)})
    up = models._Uploader(ctx, _Tensors(w))
    w = {k: np.asarray(v, np.float64) for k, v in up.source.w.items()}
    gains = [1.25, 0.75, 1.5, 0.875]
    a = R.LayerDesc(mixer=R.MIX_HEADS, norm1=up.values([gains[0]]), at_heads=4, at_kv_heads=2, at_dim=16, at_vdim=24, at_scale=0.3, at_out_scale=1.0,
                    w_q=up.matrix([("a.q", 64), ("a.k", 32), ("a.v", 48)], W), w_o=up.matrix([("a.o", W)], 96))
    r = R.LayerDesc(mixer=R.MIX_HEADS, norm1=up.values([gains[1]]), w_q=up.matrix([("r." + n, 48) for n in "qkvg"], W), w_o=up.matrix([("r.o", W)], 48))
    models._retention_heads(r, up, rt, "r")
    r.rt_out_scale = 1.0
    s = R.LayerDesc(norm1=up.values([gains[2]]), norm2=up.values([gains[3]]))
    models._mamba2_mixer(up, s, "s.", ss, W)
    s.ff_kind, s.ff_act, s.ff, s.ff_up, s.ff_down = R.FF_DENSE, R.ACT_RELU2, 40, up.matrix([("up", 40)], W), up.matrix([("down", W)], 40)
    m = _serve(ctx, R, up, [a, r, s], w, V, W, exact, 0)
    t = [int(x) for x in g.integers(0, V, 100)]
    norm = lambda x, k: P.rms(x, 1e-5) * k
    x = w["embed"][t] * 2.0
    h = norm(x, gains[0])
    q, k, v = (h @ w["a.q"].T).reshape(-1, 4, 16), (h @ w["a.k"].T).reshape(-1, 2, 16), (h @ w["a.v"].T).reshape(-1, 2, 24)
    own = np.arange(4) // 2
    p = P.softmax_visible(P.biased_scores(q, k[:, own], 0.3, np.zeros(4)), P.window_mask(100, 100))
    x = x + np.einsum("hij,jhd->ihd", p, v[:, own]).reshape(100, 96) @ w["a.o"].T
    x = x + P.retention(norm(x, gains[1]), {n: w["r." + n] for n in "qkvgo"}, rt, 1e-5)
    x = x + P.mamba2(norm(x, gains[2]), {n[2:]: w[n] for n in w if n.startswith("s.")}, ss, 1e-5)
    x = x + P.relu2_ff(norm(x, gains[3]), w["up"], w["down"])
    _check_served(m, t, P.softcap(norm(x, float(w["final"][0])) @ w["head"].T, 9.0), exact)
    m.close()


@pytest.mark.parametrize("exact", [1, 0])
def test_latent_attention_with_norms_on_the_outputs(ctx, exact):
    import runit_mac_b200 as R
    from oracle import nuvilorn as N
    from runit_mac_b200 import models
    W, V, g = 64, 70, np.random.default_rng(3)
    lin = lambda r, c: g.normal(0, 1.2 / np.sqrt(c), (r, c))
    mix = {"heads": 3, "dim": 24, "rot_dim": 8, "vdim": 16, "kv_rank": 40, "rot": {"base": 1000.0, "dims": 8}, "scale": 0.25}
    w = {"embed": lin(V, W) * 4, "head": lin(V, W) * 3, "final": g.uniform(0.5, 1.5, W), "n1": g.normal(0, 0.3, W), "n2": g.normal(0, 0.3, W)}
    w.update({"m.q": lin(96, W), "m.dkv": lin(48, W), "m.dkv.norm": g.uniform(0.5, 1.5, 40), "m.uk": lin(72, 40), "m.uv": lin(48, 40), "m.o": lin(W, 48),
              "f.gate": lin(56, W), "f.up": lin(56, W), "f.down": lin(W, 56)})
    up = models._Uploader(ctx, _Tensors(w))
    w = {k: np.asarray(v, np.float64) for k, v in up.source.w.items()}
    layers = []
    for _ in range(2):
        d = R.LayerDesc(norm1=up.gain_offset("n1", W), norm2=up.gain_offset("n2", W))
        models._latent_mixer(up, d, "m.", mix, W)
        models._dense_ff(up, d, "f.", {"ff": 56}, W)
        layers.append(d)
    m = _serve(ctx, R, up, layers, w, V, W, exact, 1)
    t = [int(x) for x in g.integers(0, V, 100)]
    x, pos = w["embed"][t] * 2.0, np.arange(100)
    mw = {n: w["m." + n] for n in ("q", "uk", "uv", "o")}
    for _ in range(2):
        x = x + P.norm_offset(N.latent_attention(x, pos, mw, mix, N.latent_of(x, pos, w["m.dkv"], w["m.dkv.norm"], mix, 1e-5)), w["n1"], 1e-5)
        x = x + P.norm_offset(N.gated_ff(x, w["f.gate"], w["f.up"], w["f.down"]), w["n2"], 1e-5)
    _check_served(m, t, P.softcap(P.norm_offset(x, w["final"] - 1, 1e-5) @ w["head"].T, 9.0), exact)
    m.close()
