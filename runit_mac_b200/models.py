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

    def beside(self, parts, rows: int) -> int:
        """Matrices side by side, as one: parts = [(name, columns)], each [rows][columns]; rows padded to pad8 of the sum."""
        out = np.zeros((rows, pad8(sum(c for _, c in parts))), np.uint16)
        at = 0
        for name, c in parts:
            out[:, at:at + c] = self._rows(name, rows, c)
            at += c
        return self._put(out)

    def gain_offset(self, name: str, n: int) -> int:
        """f32 gains of a norm whose weight is stored as the distance from one."""
        a = self.source.f32(name)
        if a.shape != (n,):
            raise ConfigError("tensor %s has shape %r, the configuration says %r" % (name, a.shape, (n,)))
        return self._put(np.float32(1.0) + a)

    def values(self, a) -> int:
        """f32 values that are computed from the configuration or from tensors."""
        return self._put(np.ascontiguousarray(a, np.float32))


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


def head_slopes(heads: int) -> np.ndarray:
    """Distance slopes of a layer's heads: a geometric series that ends at 2^-8."""
    return (2.0 ** (-8.0 * np.arange(1, heads + 1) / heads)).astype(np.float32)


def _attention_heads(d: D.LayerDesc, up: _Uploader, mix: dict):
    """Windowed attention with unit queries and keys and a distance bias per head."""
    d.at_heads, d.at_kv_heads, d.at_dim, d.at_vdim = (int(mix[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
    d.at_window, d.at_unit_qk, d.at_scale = int(mix["mask"]["size"]), 1, float(mix["scale"])
    d.at_slopes = up.values(head_slopes(d.at_heads))


def _retention_heads(d: D.LayerDesc, up: _Uploader, mix: dict, p: str):
    d.rt_heads, d.rt_dim, d.rt_vdim = (int(mix[k]) for k in ("heads", "dim", "vdim"))
    d.rt_rot_dims, d.rt_rot_base = int(mix["rot"]["dims"]), float(mix["rot"]["base"])
    decay = np.asarray(mix["decay"], np.float64)
    if decay.shape != (d.rt_heads,) or (decay < 0).any():
        raise ConfigError("%s: %d decays for %d heads, none of them negative" % (p, decay.size, d.rt_heads))
    # a decay of 0 has no logarithm: e^-1000 is 0 in f32 and stays finite when it is summed over a chunk
    d.rt_decay = up.values(np.stack([decay, np.log(np.maximum(decay, np.exp(-700.0))) - 300.0 * (decay == 0)]))


def _parallel_mixer(up: _Uploader, d: D.LayerDesc, p: str, mix: dict, width: int):
    """Attention and retention side by side on the same input; one projection in, one out."""
    left, right = mix["left"], mix["right"]
    d.mixer = D.MIX_HEADS
    _attention_heads(d, up, left)
    _retention_heads(d, up, right, p)
    d.at_out_scale, d.rt_out_scale = float(mix["left_scale"]), float(mix["right_scale"])
    L, R = p + "left.", p + "right."
    lv, rk, rv = d.at_heads * d.at_vdim, d.rt_heads * d.rt_dim, d.rt_heads * d.rt_vdim
    d.w_q = up.matrix([(L + "q", d.at_heads * d.at_dim), (L + "k", d.at_kv_heads * d.at_dim), (L + "v", d.at_kv_heads * d.at_vdim),
                       (R + "q", rk), (R + "k", rk), (R + "v", rv), (R + "g", rv)], width)
    d.w_o = up.beside([(L + "o", lv), (R + "o", rv)], width)


def _mamba2_mixer(up: _Uploader, d: D.LayerDesc, p: str, mix: dict, width: int):
    d.mixer = D.MIX_SSM
    H, vdim, N, G, taps = (int(mix[k]) for k in ("heads", "vdim", "state", "groups", "conv"))
    d.ss_heads, d.ss_vdim, d.ss_state, d.ss_groups, d.ss_taps, d.ss_norm_groups = H, vdim, N, G, taps, int(mix["norm_groups"])
    inner, channels = H * vdim, H * vdim + 2 * G * N
    d.w_q = up.matrix([(p + "in", inner + channels + H)], width)
    d.w_o = up.matrix([(p + "o", width)], inner)
    d.ss_conv, d.ss_conv_b = up.f32([p + "conv"], [(channels, taps)]), up.f32([p + "conv.b"], [(channels,)])
    d.ss_dt_bias, d.ss_skip, d.ss_norm = up.f32([p + "dt_bias"], [(H,)]), up.f32([p + "D"], [(H,)]), up.f32([p + "norm"], [(inner,)])
    a = up.source.f32(p + "A_log").astype(np.float64).reshape(-1)
    if a.size != H:
        raise ConfigError("tensor %sA_log has %d values, the configuration says %d" % (p, a.size, H))
    d.ss_a = up.values(-np.exp(a))


def _relu2_ff(up: _Uploader, d: D.LayerDesc, p: str, mlp: dict, width: int):
    d.ff_kind, d.ff_act, d.ff = D.FF_DENSE, D.ACT_RELU2, int(mlp["ff"])
    d.ff_up = up.matrix([(p + "up", d.ff)], width)
    d.ff_down = up.matrix([(p + "down", width)], d.ff)


_PAGAZEN_MIXERS = {"parallel": _parallel_mixer, "mamba2": _mamba2_mixer}


@register("Pagazen")
def build_pagazen(ctx: D.Context, cfg: dict, source, dtype: str, max_seq: int) -> D.LayeredModel:
    """Attention beside retention, or state-space layers; norms on the sublayers' outputs; layers may use another layer's
    tensors, with a cache and state of their own."""
    width, vocab = int(cfg["width"]), int(cfg["vocab"])
    up = _Uploader(ctx, source)
    entries = cfg["layers"]
    own = {}

    def layer_of(i: int) -> D.LayerDesc:
        if i in own:
            return own[i]
        layer, p, d = entries[i], "l%d." % i, D.LayerDesc()
        if layer["type"] not in _PAGAZEN_MIXERS:
            raise ConfigError("layer %d: unknown mixer %r" % (i, layer["type"]))
        d.norm1 = up.gain_offset(p + "norm1", width)
        _PAGAZEN_MIXERS[layer["type"]](up, d, p + "mix.", layer["mixer"], width)
        mlp = layer.get("mlp")
        if mlp is not None:
            if mlp["kind"] != "dense":
                raise ConfigError("layer %d: unknown feed-forward %r" % (i, mlp["kind"]))
            d.norm2 = up.gain_offset(p + "norm2", width)
            _relu2_ff(up, d, p + "mlp.", mlp, width)
        own[i] = d
        return d

    layers = []
    for i, layer in enumerate(entries):
        j = layer.get("weights_of")
        j = i if j is None else int(j)
        if not 0 <= j < len(entries) or (j != i and entries[j].get("weights_of") not in (None, j)):
            raise ConfigError("layer %d: uses the tensors of layer %d, which has none" % (i, j))
        if any(layer.get(k) != entries[j].get(k) for k in ("type", "mixer", "mlp")):
            raise ConfigError("layer %d differs from layer %d, whose tensors it uses" % (i, j))
        layers.append(layer_of(j))
    w = {"embed": up.matrix([("embed", vocab)], width), "final_norm": up.gain_offset("final.norm", width), "head": up.matrix([("head", vocab)], width)}
    c = D.LayeredCfg(n_layers=len(layers), width=width, vocab=vocab, max_seq=max_seq, exact=int(dtype == "float32"), post_norm=1,
                     eps=float(cfg["norm"]["eps"]), embed_scale=float(cfg["embedding"]["scale"]), logit_cap=float(cfg["logit_softcap"] or 0.0))
    return D.LayeredModel(ctx, c, layers, w, keep=up)


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
