"""Small Nuvilorn models with random weights for the tests (sizes chosen to reach every kernel variant)."""
import numpy as np

from oracle import nuvilorn as N


def mixer(heads, dim, rot, vdim, rank, scale=None, base=10000.0, kv_from=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "rot": {"base": base, "dims": rot},
         "scale": scale if scale is not None else (dim + rot) ** -0.5}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def config(width, vocab, layers, eps=1e-5):
    return {"architecture": "Nuvilorn", "width": width, "vocab": vocab, "norm": {"eps": eps},
            "layers": [{"type": "latent_attention", "mixer": m, "mlp": f} for m, f in layers]}


CONFIGS = {
    # every feed-forward kind, borrowed latents from two lenders, other head counts in the borrowing layers
    "mixed": config(96, 131, [(mixer(3, 24, 8, 40, 48), dense(72)), (mixer(4, 32, 8, 24, 56), moe(40, 6, 2, 56)),
                              (mixer(5, 16, 8, 48, 56, kv_from=1), moe(24, 5, 3)), (mixer(2, 40, 8, 16, 48, kv_from=0), None),
                              (mixer(3, 24, 16, 32, 32, base=500.0), moe(32, 7, 1, 16))]),
    # nothing is a multiple of eight: padded rows everywhere, prompts in the folded arrangement
    "odd": config(100, 77, [(mixer(5, 20, 6, 12, 36, base=700.0), dense(50)), (mixer(3, 10, 6, 30, 36, base=700.0, kv_from=0), moe(22, 5, 3, 30)),
                            (mixer(2, 7, 2, 9, 11), moe(13, 3, 2))], eps=1e-3),
    # more heads than a row tile, a latent that fills the wide kernels
    "wide": config(192, 300, [(mixer(20, 128, 64, 128, 272), dense(320)), (mixer(17, 64, 64, 64, 272, kv_from=0), moe(96, 12, 4, 128))]),
    # everything at its smallest
    "tiny": config(8, 16, [(mixer(1, 8, 2, 8, 8), moe(8, 1, 1, 8)), (mixer(1, 2, 2, 1, 1), dense(2))]),
    # a latent beyond 512
    "deep_latent": config(64, 50, [(mixer(2, 48, 32, 64, 600), dense(64)), (mixer(3, 96, 32, 96, 600, kv_from=0), None)]),
}


def weights(cfg, seed=0, gain=1.0):
    """Random weights; `gain` scales the projections in front of the scores."""
    g = np.random.default_rng(seed)
    W = cfg["width"]
    w = {}

    def lin(name, rows, cols, s=1.0):
        w[name] = g.normal(0, s / np.sqrt(cols), (rows, cols))

    w["embed"] = g.normal(0, 1, (cfg["vocab"], W))
    w["embed.norm"] = np.array(g.uniform(0.7, 1.4))
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = "l%d." % i, layer["mixer"], layer["mlp"]
        w[p + "norm1"], q = np.array(g.uniform(0.7, 1.4)), p + "mix."
        lin(q + "q", m["heads"] * (m["dim"] + m["rot_dim"]), W, gain)
        if m.get("kv_from") is None:
            lin(q + "dkv", m["kv_rank"] + m["rot_dim"], W)
            w[q + "dkv.norm"] = g.uniform(0.5, 1.5, m["kv_rank"])
        lin(q + "uk", m["heads"] * m["dim"], m["kv_rank"])
        lin(q + "uv", m["heads"] * m["vdim"], m["kv_rank"])
        lin(q + "o", W, m["heads"] * m["vdim"], 1.5)
        if f is None:
            continue
        w[p + "norm2"], q = np.array(g.uniform(0.7, 1.4)), p + "mlp."
        if f["kind"] == "dense":
            for n in ("gate", "up"):
                lin(q + n, f["ff"], W, 1.5)
            lin(q + "down", W, f["ff"], 1.5)
            continue
        lin(q + "router", f["router"]["experts"], W, 2.0)
        for e in range(f["router"]["experts"]):
            lin(q + "e%d.up" % e, f["expert"]["ff"], W, 1.5)
            lin(q + "e%d.down" % e, W, f["expert"]["ff"], 1.5)
        if f.get("shared"):
            lin(q + "shared.up", f["shared"]["ff"], W, 1.5)
            lin(q + "shared.down", W, f["shared"]["ff"], 1.5)
            lin(q + "shared.sg", 1, W, 2.0)
    w["final.norm"] = np.array(g.uniform(0.7, 1.4))
    lin("head", cfg["vocab"], W, 2.0)
    return w


def folder(path, cfg, seed=0, gain=1.0, edit=None):
    """Writes a model folder; returns the weights as the file holds them."""
    w = weights(cfg, seed, gain)
    if edit:
        edit(w)
    return N.save_folder(path, cfg, w)


def tokens(cfg, n, seed=1):
    return [int(t) for t in np.random.default_rng(seed).integers(0, cfg["vocab"], n)]


def greedy(cfg, w, prompt, n):
    """Greedy continuation by the plain implementation (whole sequence again for every token)."""
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(np.argmax(N.forward(cfg, w, seq)[-1])))
    return seq[len(prompt):]


def row_errors(got, ref):
    """Root mean square difference per row (mean taken off), relative to the spread of the reference."""
    d = np.asarray(got, np.float64) - ref
    d -= d.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / np.std(ref)


def routing_margins(cfg, w, toks):
    """Per token the smallest distance, over the layers, between the logits of the last chosen and the first left-out expert."""
    out = np.full(len(toks), np.inf)
    real = N.route_sigmoid

    def watch(h, w_router, top):
        z = -np.sort(-(h @ w_router.T), axis=-1)
        if top < z.shape[1]:
            out[:] = np.minimum(out, z[:, top - 1] - z[:, top])
        return real(h, w_router, top)
    N.route_sigmoid = watch
    try:
        N.forward(cfg, w, toks)
    finally:
        N.route_sigmoid = real
    return out
