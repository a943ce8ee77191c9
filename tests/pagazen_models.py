"""Small Pagazen models with random weights for the tests (sizes chosen to reach every kernel variant)."""
import numpy as np

from oracle import pagazen as P
from nuvilorn_models import row_errors, tokens  # noqa: F401


def left(heads, kv, dim, vdim, window, scale=None):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "mask": {"size": window}, "scale": scale if scale is not None else dim ** -0.5}


def right(heads, dim, vdim, rot, base=10000.0, decay=None):
    if decay is None:
        decay = [float(1 - 2.0 ** -(2 + 2 * h)) for h in range(heads)]
    return {"heads": heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot}, "decay": decay}


def parallel(lf, rt, ls=0.8, rs=0.7):
    return {"type": "parallel", "mixer": {"left": lf, "right": rt, "left_scale": ls, "right_scale": rs}}


def mamba(heads, vdim, state, groups=1, conv=4, norm_groups=1):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}}


def config(width, vocab, layers, scale=3.0, cap=12.0, eps=1e-5):
    """layers: (mixer entry, ff or None), or the number of the layer whose tensors are used."""
    out = []
    for item in layers:
        if isinstance(item, int):
            out.append(dict(out[item], weights_of=item))
        else:
            entry, ff = item
            out.append(dict(entry, mlp=None if ff is None else {"kind": "dense", "ff": ff}))
    return {"architecture": "Pagazen", "width": width, "vocab": vocab, "embedding": {"scale": scale}, "norm": {"eps": eps}, "logit_softcap": cap,
            "layers": out}


CONFIGS = {
    # both mixers, partial rotation, several groups, layers that use another layer's tensors, a layer without feed-forward
    "mixed": config(80, 131, [(parallel(left(6, 3, 40, 24, 37), right(3, 32, 48, 20)), 72), (mamba(6, 16, 40, groups=3, conv=5, norm_groups=2), 56), 0,
                              (mamba(4, 24, 16, norm_groups=1), None), 1, (parallel(left(2, 2, 16, 16, 9), right(2, 16, 8, 16, base=300.0), 1.3, 0.4), 40)]),
    # nothing is a multiple of eight, norm groups that cut through heads, a window of five
    "odd": config(50, 77, [(mamba(3, 5, 6, conv=2, norm_groups=5), 30), (parallel(left(5, 1, 11, 9, 5), right(2, 10, 7, 6, base=70.0, decay=[0.9, 1.0])), 45),
                           (mamba(2, 3, 7, groups=2, conv=3, norm_groups=1), 21)], eps=1e-3),
    # two blocks of query heads per key head, key dimensions beyond 128, wide states
    "wide": config(192, 300, [(parallel(left(16, 1, 128, 64, 200), right(2, 256, 160, 256)), 320), (mamba(4, 64, 128, groups=2, norm_groups=2), 256), 1]),
    # everything at its smallest: a window of one, one tap
    "tiny": config(8, 16, [(parallel(left(1, 1, 1, 1, 1), right(1, 2, 1, 2, decay=[0.5])), 3), (mamba(1, 1, 1, conv=1), 2)]),
    # sizes past the tensor-core kernels: heads of 200, keys of 300
    "large_keys": config(64, 50, [(parallel(left(2, 1, 200, 208, 70), right(2, 300, 40, 100)), 64), (mamba(2, 40, 280, conv=6), 48)]),
}


def weights(cfg, seed=0, gain=1.0):
    """Random weights; `gain` scales the projections in front of the scores."""
    g = np.random.default_rng(seed)
    W, w = cfg["width"], {}

    def lin(name, rows, cols, s=1.0):
        w[name] = g.normal(0, s / np.sqrt(cols), (rows, cols))

    lin("embed", cfg["vocab"], W, np.sqrt(W) / cfg["embedding"]["scale"])
    for i, layer in enumerate(cfg["layers"]):
        if "weights_of" in layer:
            continue
        p, m = "l%d." % i, layer["mixer"]
        q = p + "mix."
        w[p + "norm1"] = g.normal(0, 0.3, W)
        if layer["type"] == "parallel":
            a, r = m["left"], m["right"]
            for n, rows in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])):
                lin(q + "left." + n, rows, W)
            lin(q + "left.o", W, a["heads"] * a["vdim"])
            for n, rows in (("q", r["heads"] * r["dim"]), ("k", r["heads"] * r["dim"]), ("v", r["heads"] * r["vdim"]), ("g", r["heads"] * r["vdim"])):
                lin(q + "right." + n, rows, W, gain if n in "qk" else 1.0)
            lin(q + "right.o", W, r["heads"] * r["vdim"])
        else:
            H, inner, gn = m["heads"], m["heads"] * m["vdim"], m["groups"] * m["state"]
            ch = inner + 2 * gn
            lin(q + "in", inner + ch + H, W, gain)
            w[q + "conv"], w[q + "conv.b"] = g.normal(0, 1 / np.sqrt(m["conv"]), (ch, m["conv"])), g.normal(0, 0.2, ch)
            w[q + "dt_bias"], w[q + "A_log"] = g.uniform(-4, 0, H), g.uniform(-1.5, 1.5, H)
            w[q + "D"], w[q + "norm"] = g.normal(0, 1, H), g.uniform(0.5, 1.5, inner)
            lin(q + "o", W, inner)
        if layer["mlp"] is not None:
            w[p + "norm2"] = g.normal(0, 0.3, W)
            lin(p + "mlp.up", layer["mlp"]["ff"], W)
            lin(p + "mlp.down", W, layer["mlp"]["ff"])
    w["final.norm"] = g.normal(0, 0.3, W)
    lin("head", cfg["vocab"], W, 4.0)
    return w


def folder(path, cfg, seed=0, gain=1.0, edit=None):
    """Writes a model folder; returns the weights as the file holds them."""
    w = weights(cfg, seed, gain)
    if edit:
        edit(w)
    return P.save_folder(path, cfg, w)


def greedy(cfg, w, prompt, n):
    """Greedy continuation by the plain implementation (whole sequence again for every token)."""
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(np.argmax(P.forward(cfg, w, seq)[-1])))
    return seq[len(prompt):]
