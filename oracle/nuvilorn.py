"""Plain numpy restatement of the Nuvilorn decoder: one function per mechanism, whole sequences at a time, no cache.

Test infrastructure only.  Everything is computed in float64 from the values the tensors hold; nothing here is shared
with the library.  Weights are a dict of numpy arrays under the tensor names of a model folder; `cfg` is the parsed
config.json.
"""
from __future__ import annotations

import json
import struct
from pathlib import Path

import numpy as np


# ── mechanisms ──
def rms(x, eps):
    """x divided by its root mean square over the last axis (eps inside the root)."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm_scalar(x, g, eps):
    """RMS norm with one gain for all coordinates."""
    return rms(x, eps) * float(np.asarray(g).reshape(()))


def rms_norm(x, weight, eps):
    """RMS norm with a gain per coordinate."""
    return rms(x, eps) * weight


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def rotate_interleaved(x, pos, dims, base):
    """Rotary positions on the first `dims` coordinates of the last axis; coordinates 2i and 2i+1 form a pair.
    x: [tokens, ..., d], pos: [tokens]."""
    out = np.array(x, np.float64)
    i = np.arange(dims // 2)
    a = np.asarray(pos, np.float64)[:, None] * float(base) ** (-2.0 * i / dims)
    shape = (len(pos),) + (1,) * (x.ndim - 2) + (dims // 2,)
    c, s = np.cos(a).reshape(shape), np.sin(a).reshape(shape)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def latent_of(h, pos, w_dkv, norm_w, mix, eps):
    """(normed latent [n, kv_rank], rotated shared key part [n, rot_dim]) of a layer that has its own projection."""
    y = h @ w_dkv.T
    r = mix["kv_rank"]
    return rms_norm(y[:, :r], norm_w, eps), rotate_interleaved(y[:, r:], pos, mix["rot_dim"], mix["rot"]["base"])


def causal_softmax(scores):
    """Row i of the last two axes sees columns j <= i."""
    n = scores.shape[-1]
    s = np.where(np.tril(np.ones((n, n), bool)), scores, -np.inf)
    p = np.exp(s - s.max(-1, keepdims=True))
    return p / p.sum(-1, keepdims=True)


def latent_attention(h, pos, w, mix, latent):
    """w: dict with q, uk, uv, o; latent = (c, k_rot) of this layer or of the one it borrows from."""
    n, H, d, r, dv = len(h), mix["heads"], mix["dim"], mix["rot_dim"], mix["vdim"]
    c, k_rot = latent
    q = (h @ w["q"].T).reshape(n, H, d + r)
    q_un, q_rot = q[..., :d], rotate_interleaved(q[..., d:], pos, r, mix["rot"]["base"])
    k_un = (c @ w["uk"].T).reshape(n, H, d)
    v = (c @ w["uv"].T).reshape(n, H, dv)
    s = np.einsum("ihd,jhd->hij", q_un, k_un) + np.einsum("ihd,jd->hij", q_rot, k_rot)
    p = causal_softmax(s * mix["scale"])
    return np.einsum("hij,jhd->ihd", p, v).reshape(n, H * dv) @ w["o"].T


def gated_ff(h, w_gate, w_up, w_down):
    g = h @ w_gate.T
    return (g * sigmoid(g) * (h @ w_up.T)) @ w_down.T


def relu2_ff(h, w_up, w_down):
    return np.square(np.maximum(h @ w_up.T, 0.0)) @ w_down.T


def route_sigmoid(h, w_router, top):
    """(expert ids [n, top] by falling score, their scores)."""
    s = sigmoid(h @ w_router.T)
    idx = np.argsort(-s, axis=-1, kind="stable")[:, :top]
    return idx, np.take_along_axis(s, idx, -1)


def moe(h, w, mlp):
    """w: dict of the layer's mlp tensors.  The routing weight scales an expert's input; the shared expert's output is
    scaled by the sigmoid of its own gate row."""
    idx, s = route_sigmoid(h, w["router"], mlp["router"]["top"])
    out = np.zeros_like(h)
    for t in range(len(h)):
        for e, a in zip(idx[t], s[t]):
            out[t] += relu2_ff(a * h[t], w["e%d.up" % e], w["e%d.down" % e])
    if mlp.get("shared"):
        out += sigmoid(h @ w["shared.sg"].T) * relu2_ff(h, w["shared.up"], w["shared.down"])
    return out


# ── the model ──
def _sub(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def forward(cfg, weights, tokens, want_layers=False):
    """Logits [n, vocab] of one sequence (and the residual stream after every layer)."""
    w = {k: np.asarray(v, np.float64) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    pos = np.arange(len(tokens))
    x = rms_norm_scalar(w["embed"][np.asarray(tokens)], w["embed.norm"], eps)
    latents, trail = {}, []
    for i, layer in enumerate(cfg["layers"]):
        p, mix, mlp = "l%d." % i, layer["mixer"], layer["mlp"]
        m = _sub(w, p + "mix.")
        h = rms_norm_scalar(x, w[p + "norm1"], eps)
        src = mix.get("kv_from")
        if src is None:
            latents[i] = latent_of(h, pos, m["dkv"], m["dkv.norm"], mix, eps)
            src = i
        x = x + latent_attention(h, pos, m, mix, latents[src])
        if mlp is not None:
            h = rms_norm_scalar(x, w[p + "norm2"], eps)
            f = _sub(w, p + "mlp.")
            x = x + (gated_ff(h, f["gate"], f["up"], f["down"]) if mlp["kind"] == "dense" else moe(h, f, mlp))
        trail.append(x)
    logits = rms_norm_scalar(x, w["final.norm"], eps) @ w["head"].T
    return (logits, np.stack(trail)) if want_layers else logits


# ── model folders ──
def to_bf16(x):
    """Round to bfloat16 (to nearest, ties to even); returns the uint16 patterns."""
    b = np.ascontiguousarray(x, np.float32).view(np.uint32).astype(np.uint64)
    return ((b + 0x7FFF + ((b >> 16) & 1)) >> 16).astype(np.uint16)


def from_bf16(u):
    return (np.asarray(u, np.uint16).astype(np.uint32) << 16).view(np.float32)


def save_folder(path, cfg, weights):
    """config.json and model.safetensors (bfloat16) of a model; returns the weights as the file holds them."""
    path = Path(path)
    path.mkdir(parents=True, exist_ok=True)
    head, blobs, off, kept = {}, [], 0, {}
    for name, a in weights.items():
        a = np.asarray(a, np.float32)
        u = to_bf16(a).reshape(a.shape)
        b = u.tobytes()
        head[name] = {"dtype": "BF16", "shape": list(a.shape), "data_offsets": [off, off + len(b)]}
        off += len(b)
        blobs.append(b)
        kept[name] = from_bf16(u)
    hj = json.dumps(head).encode()
    with open(path / "model.safetensors", "wb") as f:
        f.write(struct.pack("<Q", len(hj)) + hj)
        for b in blobs:
            f.write(b)
    (path / "config.json").write_text(json.dumps(cfg))
    return kept


def load_folder(path):
    path = Path(path)
    raw = (path / "model.safetensors").read_bytes()
    n = struct.unpack("<Q", raw[:8])[0]
    out = {}
    for name, t in json.loads(raw[8:8 + n]).items():
        if name != "__metadata__":
            a, b = t["data_offsets"]
            out[name] = from_bf16(np.frombuffer(raw[8 + n + a:8 + n + b], np.uint16)).reshape(t["shape"])
    return json.loads((path / "config.json").read_text()), out
