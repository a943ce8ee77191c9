"""Plain numpy restatement of the Pagazen decoder: one function per mechanism, whole sequences at a time, no cache.

Test infrastructure only.  Everything is computed in float64 from the values the tensors hold, recurrences token by token;
nothing here is shared with the library.  Weights are a dict of numpy arrays under the tensor names of a model folder; `cfg`
is the parsed config.json.
"""
from __future__ import annotations

import numpy as np

from .nuvilorn import load_folder, rms, save_folder, sigmoid  # noqa: F401


# ── mechanisms ──
def norm_offset(x, w, eps):
    """RMS norm with a gain per coordinate that is stored as its distance from one."""
    return rms(x, eps) * (1.0 + w)


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def softcap(z, cap):
    return cap * np.tanh(z / cap)


def head_slopes(heads):
    """Distance slope of every head: a geometric series that ends at 2^-8."""
    return 2.0 ** (-8.0 * np.arange(1, heads + 1) / heads)


def rotate_halves(x, pos, dims, base):
    """Rotary positions on the first `dims` coordinates of the last axis; coordinates i and i + dims/2 form a pair.
    x: [tokens, heads, d]."""
    out = np.array(x, np.float64)
    half = dims // 2
    a = np.asarray(pos, np.float64)[:, None] * float(base) ** (-2.0 * np.arange(half) / dims)
    c, s = np.cos(a)[:, None, :], np.sin(a)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    out[..., :half] = u * c - v * s
    out[..., half:dims] = v * c + u * s
    return out


def window_mask(n, size):
    """[i, j]: position i sees itself and the size - 1 positions before it."""
    d = np.arange(n)[:, None] - np.arange(n)[None, :]
    return (d >= 0) & (d < size)


def biased_scores(q, k, scale, slopes):
    """[heads, i, j]: scaled products less slope * distance.  q, k: [n, heads, dim]."""
    n = len(q)
    d = np.arange(n)[:, None] - np.arange(n)[None, :]
    return np.einsum("ihd,jhd->hij", q, k) * scale - np.asarray(slopes)[:, None, None] * d


def softmax_visible(s, visible):
    s = np.where(visible, s, -np.inf)
    p = np.exp(s - s.max(-1, keepdims=True))
    return p / p.sum(-1, keepdims=True)


def window_attention(h, w, mix, eps):
    """Grouped-query attention over a sliding window, queries and keys of unit root mean square; w: q, k, v, o."""
    n, H, G, d, dv = len(h), mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    q = rms((h @ w["q"].T).reshape(n, H, d), eps)
    k = rms((h @ w["k"].T).reshape(n, G, d), eps)
    v = (h @ w["v"].T).reshape(n, G, dv)
    own = np.arange(H) // (H // G)
    s = biased_scores(q, k[:, own], mix["scale"], head_slopes(H))
    p = softmax_visible(s, window_mask(n, mix["mask"]["size"]))
    return np.einsum("hij,jhd->ihd", p, v[:, own]).reshape(n, H * dv) @ w["o"].T


def linear_scan(q, k, v, decay):
    """S_t = decay_t S_(t-1) + k_t v_t^T, o_t = S_t^T q_t per head.  q, k: [n, heads, dk], v: [n, heads, dv],
    decay: [n, heads]."""
    n, H, dk = k.shape
    S = np.zeros((H, dk, v.shape[2]))
    out = np.zeros((n, H, v.shape[2]))
    for t in range(n):
        S = decay[t][:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hkv,hk->hv", S, q[t])
    return out


def retention(h, w, mix, eps):
    """Linear attention with a fixed decay per head, rotary positions and a gate; w: q, k, v, g, o."""
    n, H, d, dv = len(h), mix["heads"], mix["dim"], mix["vdim"]
    pos, rot = np.arange(n), mix["rot"]
    q = rotate_halves((h @ w["q"].T).reshape(n, H, d), pos, rot["dims"], rot["base"])
    k = rotate_halves((h @ w["k"].T).reshape(n, H, d), pos, rot["dims"], rot["base"]) * d ** -0.5
    v = (h @ w["v"].T).reshape(n, H, dv)
    o = linear_scan(q, k, v, np.broadcast_to(np.asarray(mix["decay"], np.float64), (n, H)))
    return (rms(o, eps).reshape(n, H * dv) * silu(h @ w["g"].T)) @ w["o"].T


def parallel(h, w, mix, eps):
    left = window_attention(h, _sub(w, "left."), mix["left"], eps)
    right = retention(h, _sub(w, "right."), mix["right"], eps)
    return mix["left_scale"] * left + mix["right_scale"] * right


def causal_conv(x, w, b):
    """Per channel; the last column of w is the current token's, zeros stand before the start.  x: [n, channels]."""
    taps = w.shape[1]
    y = np.zeros_like(x)
    for j in range(taps):
        back = taps - 1 - j
        if back < len(x):
            y[back:] += w[:, j] * x[:len(x) - back]
    return y + b


def mamba2(h, w, mix, eps):
    """State-space layer with a scalar decay per head and token; w: in, conv, conv.b, dt_bias, A_log, D, norm, o."""
    n, H, dv, N, G = len(h), mix["heads"], mix["vdim"], mix["state"], mix["groups"]
    inner = H * dv
    z, xbc, dt = np.split(h @ w["in"].T, [inner, 2 * inner + 2 * G * N], axis=1)
    xbc = silu(causal_conv(xbc, w["conv"], w["conv.b"]))
    x, B, C = np.split(xbc, [inner, inner + G * N], axis=1)
    x, own = x.reshape(n, H, dv), np.arange(H) // (H // G)
    B, C = B.reshape(n, G, N)[:, own], C.reshape(n, G, N)[:, own]
    dt = softplus(dt + w["dt_bias"])
    y = linear_scan(C, B * dt[..., None], x, np.exp(-np.exp(w["A_log"]) * dt)) + w["D"][:, None] * x
    y = y.reshape(n, inner) * silu(z)
    y = rms(y.reshape(n, mix["norm_groups"], -1), eps).reshape(n, inner) * w["norm"]
    return y @ w["o"].T


def relu2_ff(h, w_up, w_down):
    return np.square(np.maximum(h @ w_up.T, 0.0)) @ w_down.T


MIXERS = {"parallel": lambda h, w, mix, eps: parallel(h, w, mix, eps), "mamba2": lambda h, w, mix, eps: mamba2(h, w, mix, eps)}


# ── the model ──
def _sub(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def forward(cfg, weights, tokens, want_layers=False):
    """Logits [n, vocab] of one sequence (and the residual stream after every layer)."""
    w = {k: np.asarray(v, np.float64) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    trail = []
    for i, layer in enumerate(cfg["layers"]):
        p = "l%d." % layer.get("weights_of", i)
        x = x + norm_offset(MIXERS[layer["type"]](x, _sub(w, p + "mix."), layer["mixer"], eps), w[p + "norm1"], eps)
        if layer["mlp"] is not None:
            f = _sub(w, p + "mlp.")
            x = x + norm_offset(relu2_ff(x, f["up"], f["down"]), w[p + "norm2"], eps)
        trail.append(x)
    logits = softcap(norm_offset(x, w["final.norm"], eps) @ w["head"].T, cfg["logit_softcap"])
    return (logits, np.stack(trail)) if want_layers else logits
