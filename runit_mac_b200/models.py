"""Model registry: architecture name of a model folder (config.json + model.safetensors) -> the decoder that serves it.

An architecture is a function ``build(ctx, cfg, source, dtype, max_seq) -> Model`` registered under the name config.json
gives in ``architecture``.  ``source`` hands out tensors by name (a SafetensorsFile).  The OLMoE-shaped Q4_K decoder is
built from packed device buffers (``Model`` in dispatch.py, weights through gguf.py).
"""
from __future__ import annotations

import json
from pathlib import Path

import numpy as np

from . import dispatch as D
from .safetensors import SafetensorsFile

ARCHITECTURES = {}
DTYPES = ("bfloat16", "float32")


class ConfigError(ValueError):
    pass


def register(name: str):
    def wrap(fn):
        ARCHITECTURES[name] = fn
        return fn
    return wrap


def load_config(path) -> dict:
    return json.loads((Path(path) / "config.json").read_text())


def load_model(ctx: D.Context, path, dtype: str = "bfloat16", max_seq: int = 4096) -> D.Model:
    """The decoder of a model folder, weights on the device.  dtype: "bfloat16" (how the model is served) or "float32"
    (activations and cache in 32-bit throughout)."""
    if dtype not in DTYPES:
        raise ConfigError("dtype %r (one of %s)" % (dtype, ", ".join(DTYPES)))
    cfg = load_config(path)
    name = cfg.get("architecture")
    if name not in ARCHITECTURES:
        raise ConfigError("unknown architecture %r (known: %s)" % (name, ", ".join(sorted(ARCHITECTURES))))
    return ARCHITECTURES[name](ctx, cfg, SafetensorsFile(Path(path) / "model.safetensors"), dtype, max_seq)


# ── device layouts of the layered decoders (runit_layer_desc) ──
def pad8(n: int) -> int:
    return (n + 7) // 8 * 8


class _Uploader:
    """Uploads tensors in the layouts of the layered decoders and owns the buffers."""

    def __init__(self, ctx: D.Context, source):
        self.ctx, self.source, self.buffers = ctx, source, []

    def _put(self, a: np.ndarray) -> int:
        b = self.ctx.buffer_from(a)
        self.buffers.append(b)
        return b.ptr

    def _rows(self, name: str, rows: int, cols: int) -> np.ndarray:
        if self.source.shape(name) != (rows, cols):
            raise ConfigError("tensor %s has shape %r, the configuration says %r" % (name, self.source.shape(name), (rows, cols)))
        return self.source.bf16(name)

    def matrix(self, parts, cols: int) -> int:
        """Matrices under one another, as one: parts = [(name, rows)], each [rows][cols]; rows padded to pad8(cols)."""
        out = np.zeros((sum(r for _, r in parts), pad8(cols)), np.uint16)
        at = 0
        for name, r in parts:
            out[at:at + r, :cols] = self._rows(name, r, cols)
            at += r
        return self._put(out)

    def gated(self, gate: str, up: str, rows: int, cols: int) -> int:
        """Gate and up rows interleaved: row 2i = gate i, row 2i+1 = up i."""
        out = np.zeros((2 * rows, pad8(cols)), np.uint16)
        out[0::2, :cols] = self._rows(gate, rows, cols)
        out[1::2, :cols] = self._rows(up, rows, cols)
        return self._put(out)

    def f32(self, names, shape) -> int:
        """f32 values, tensors one after the other; shape is that of each."""
        parts = []
        for n, s in zip(names, shape):
            a = self.source.f32(n)
            if int(np.prod(s, dtype=np.int64)) != a.size:
                raise ConfigError("tensor %s has shape %r, the configuration says %r" % (n, self.source.shape(n), s))
            parts.append(a.reshape(-1))
        return self._put(np.concatenate(parts))


def _latent_mixer(up: _Uploader, d: D.LayerDesc, p: str, mix: dict, width: int):
    """Latent attention: mixer sizes and tensors of the layer with prefix p."""
    H, dim, rot, vdim, rank = (int(mix[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    if int(mix["rot"]["dims"]) != rot:
        raise ConfigError("%s: the rotated part has %d dimensions, %d of them rotate" % (p, rot, mix["rot"]["dims"]))
    d.heads, d.dim, d.rot_dim, d.vdim, d.kv_rank = H, dim, rot, vdim, rank
    d.scale, d.rot_base = float(mix["scale"]), float(mix["rot"]["base"])
    src = mix.get("kv_from")
    d.kv_from = -1 if src is None else int(src)
    q = [(p + "q", H * (dim + rot))]
    if src is None:
        q.append((p + "dkv", rank + rot))
        d.kv_norm = up.f32([p + "dkv.norm"], [(rank,)])
    d.w_q = up.matrix(q, width)
    d.w_ukv = up.matrix([(p + "uk", H * dim), (p + "uv", H * vdim)], rank)
    d.w_o = up.matrix([(p + "o", width)], H * vdim)


def _dense_ff(up: _Uploader, d: D.LayerDesc, p: str, mlp: dict, width: int):
    d.ff_kind, d.ff_act, d.ff = D.FF_DENSE, D.ACT_SILU_GLU, int(mlp["ff"])
    d.ff_up = up.gated(p + "gate", p + "up", d.ff, width)
    d.ff_down = up.matrix([(p + "down", width)], d.ff)


def _moe_ff(up: _Uploader, d: D.LayerDesc, p: str, mlp: dict, width: int):
    E, ff = int(mlp["router"]["experts"]), int(mlp["expert"]["ff"])
    d.ff_kind, d.ff_act, d.ff = D.FF_MOE, D.ACT_RELU2, ff
    d.n_experts, d.top_k, d.score, d.renorm = E, int(mlp["router"]["top"]), D.SCORE_SIGMOID, 0
    d.ff_up = up.matrix([(p + "e%d.up" % e, ff) for e in range(E)], width)
    d.ff_down = up.matrix([(p + "e%d.down" % e, width) for e in range(E)], ff)
    shared = mlp.get("shared")
    rows, shapes = [p + "router"], [(E, width)]
    if shared:
        d.shared_ff = int(shared["ff"])
        d.shared_up = up.matrix([(p + "shared.up", d.shared_ff)], width)
        d.shared_down = up.matrix([(p + "shared.down", width)], d.shared_ff)
        rows.append(p + "shared.sg")
        shapes.append((1, width))
    d.router = up.f32(rows, shapes)


@register("Nuvilorn")
def build_nuvilorn(ctx: D.Context, cfg: dict, source, dtype: str, max_seq: int) -> D.LayeredModel:
    """Latent attention with borrowed latents, dense or mixture-of-experts feed-forward, norms with one gain."""
    width, vocab = int(cfg["width"]), int(cfg["vocab"])
    up = _Uploader(ctx, source)
    layers = []
    for i, layer in enumerate(cfg["layers"]):
        p = "l%d." % i
        d = D.LayerDesc()
        if layer["type"] != "latent_attention":
            raise ConfigError("layer %d: unknown mixer %r" % (i, layer["type"]))
        d.norm1 = up.f32([p + "norm1"], [()])
        _latent_mixer(up, d, p + "mix.", layer["mixer"], width)
        mlp = layer.get("mlp")
        if mlp is not None:
            d.norm2 = up.f32([p + "norm2"], [()])
            if mlp["kind"] == "dense":
                _dense_ff(up, d, p + "mlp.", mlp, width)
            elif mlp["kind"] == "moe":
                _moe_ff(up, d, p + "mlp.", mlp, width)
            else:
                raise ConfigError("layer %d: unknown feed-forward %r" % (i, mlp["kind"]))
        layers.append(d)
    w = {"embed": up.matrix([("embed", vocab)], width), "embed_norm": up.f32(["embed.norm"], [()]),
         "final_norm": up.f32(["final.norm"], [()]), "head": up.matrix([("head", vocab)], width)}
    c = D.LayeredCfg(n_layers=len(layers), width=width, vocab=vocab, max_seq=max_seq, exact=int(dtype == "float32"),
                     eps=float(cfg["norm"]["eps"]))
    return D.LayeredModel(ctx, c, layers, w, keep=up)
