"""Small Palulorn configurations and weights for the tests (not the product's generator: shapes are derived here from the
config, so the product's own shape table is checked against this one)."""
import math

import torch


def moe(ff, experts, top, count=1, keep=1, scale=1.0, shared=None):
    r = {"experts": experts, "top": top, "scale": scale}
    if count > 1:
        r["groups"] = {"count": count, "keep": keep}
    f = {"kind": "moe", "expert": {"ff": ff}, "router": r}
    if shared:
        f["shared"] = {"ff": shared}
    return f


def left(heads, kv_heads, dim, coef=0.3, every=16, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale or 1.0 / math.sqrt(dim)}
    if every:
        m["q_temp"] = {"coef": coef, "every": every}
    return m


def pair(a, heads, dim, vdim, cap=6.0):
    return {"type": "parallel", "mixer": {"left": a, "right": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}}


def rglru(width, blocks, conv=4):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}}


def attention(heads, kv_heads, dim, vdim, window, rot_dims, base=100.0, factor=None, conv=4, scale=None):
    rot = {"base": base, "dims": rot_dims}
    if factor:
        rot["scaling"] = {"factor": factor}
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "rot": rot,
         "scale": scale or 1.0 / math.sqrt(dim)}
    if window:
        m["mask"] = {"size": window}
    return {"type": "attention", "mixer": m}


def config(layers, width=64, vocab=97, eps=1e-5, embed_scale=3.0, loop=None):
    """layers: list of (mixer entry, feed-forward entry or None); loop: (start, stop, times) or None."""
    c = {"architecture": "Palulorn", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": embed_scale},
         "layers": [dict(m, mlp=f) for m, f in layers]}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


def shapes(cfg):
    W, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
    if "loop" in cfg:
        out["loop.in"], out["loop.step"] = (W, 2 * W), (cfg["loop"]["times"], W)
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        out[p + "norm1"] = (W,)
        if L["type"] == "parallel":
            a, b = m["left"], m["right"]
            H, G, d = a["heads"], a["kv_heads"], a["dim"]
            q = p + "mix.left."
            out.update({q + "q": (H * d, W), q + "q.b": (H * d,), q + "k": (G * d, W), q + "k.b": (G * d,), q + "sink": (H,),
                        q + "g": (H, W), q + "o": (W, H * d), q + "o.b": (W,), q + "out": (W,)})
            H, d, v = b["heads"], b["dim"], b["vdim"]
            q = p + "mix.right."
            out.update({q + "q": (H * d, W), q + "k": (H * d, W), q + "v": (H * v, W), q + "g": (H * v, W),
                        q + "o": (W, H * v), q + "norm": (H * v,), q + "i": (H, W), q + "i.b": (H,), q + "f": (H, W),
                        q + "f.b": (H,), q + "out": (W,)})
        elif L["type"] == "rglru":
            n, nb, q = m["width"], m["blocks"], p + "mix."
            out.update({q + "y": (n, W), q + "y.b": (n,), q + "x": (n, W), q + "x.b": (n,), q + "conv": (n, m["conv"]),
                        q + "conv.b": (n,), q + "lam": (n,), q + "o": (W, n)})
            for r in ("ra", "ri"):
                out.update({q + r: (nb, n // nb, n // nb), q + r + ".b": (nb, n // nb)})
        else:
            q = p + "mix."
            for c, n in (("q", m["heads"] * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"])):
                out.update({q + c: (n, W), q + c + ".b": (n,), q + c + ".conv": (n, m["conv"])})
            out.update({q + "q.norm": (m["dim"],), q + "k.norm": (m["dim"],), q + "o": (W, m["heads"] * m["vdim"])})
        f = L["mlp"]
        if f is not None:
            q = p + "mlp."
            out[p + "norm2"], out[q + "router"] = (W,), (f["router"]["experts"], W)
            for e in range(f["router"]["experts"]):
                out.update({q + f"e{e}.up": (f["expert"]["ff"], W), q + f"e{e}.down": (W, f["expert"]["ff"])})
            if "shared" in f:
                out.update({q + "shared.up": (f["shared"]["ff"], W), q + "shared.down": (W, f["shared"]["ff"])})
    return out


def weights(cfg, seed=0, alike=0.0):
    """bf16 tensors: projections N(0, 1/in); keys, sinks and key gains large enough that attention is sharp and a wrong key,
    a lost sink or a window that is off by one shows; forget gates and decays from nearly forgetful to nearly lossless.
    alike: share of every expert that all experts of a layer have in common (with a choice that rounding may turn over)."""
    g = torch.Generator().manual_seed(seed)
    out, common = {}, {}
    for name, shp in shapes(cfg).items():
        leaf = name.split(".")[-1]
        r = torch.randn(shp, generator=g)
        if leaf in ("norm1", "norm2", "out"):
            t = 1.0 + 0.3 * r
        elif name.endswith((".k.norm", ".q.norm")):
            t = 1.6 + 0.3 * r
        elif leaf == "norm":
            t = 1.0 + 0.3 * r
        elif name.endswith(("left.q", "left.k")):
            t = 1.7 * r / math.sqrt(shp[-1])
        elif leaf == "sink":
            t = 1.0 + r
        elif name.endswith("right.f.b"):
            t = 2.0 + 2.0 * r
        elif leaf == "lam":
            t = -3.0 + 1.5 * r
        elif leaf == "conv":
            t = r / math.sqrt(shp[-1])
        elif leaf == "router":
            t = 2.0 * r / math.sqrt(shp[-1])
        elif name == "embed":
            t = r / math.sqrt(shp[-1])
        elif len(shp) == 1 or leaf in ("b", "step"):
            t = 0.5 * r
        else:
            t = r / math.sqrt(shp[-1])
        if alike and ".mlp.e" in name:
            layer = name.split(".mlp.")[0] + leaf
            common.setdefault(layer, t)
            t = alike * common[layer] + math.sqrt(1.0 - alike * alike) * t
        out[name] = t.to(torch.bfloat16)
    return out


def row_errors(got, want):
    """Per row: root mean square of the difference of the mean-free logits over that of the wanted ones."""
    got, want = got.double().cpu(), want.double().cpu()
    got = got - got.mean(dim=-1, keepdim=True)
    want = want - want.mean(dim=-1, keepdim=True)
    return (got - want).pow(2).mean(dim=-1).sqrt() / want.pow(2).mean(dim=-1).sqrt()


CONFIGS = {
    # all mixers, a loop in the middle, sizes that differ from each other on every side
    "mix": config([
        (rglru(40, 5, conv=3), moe(24, 6, 2, 3, 2, scale=1.5, shared=20)),
        (pair(left(4, 2, 12), 3, 20, 16), moe(16, 8, 3, 2, 1, scale=2.0, shared=32)),
        (attention(6, 3, 16, 8, 13, 8, factor=3.0), None),
        (pair(left(5, 1, 16, every=0), 2, 12, 20, cap=9.0), None),
    ], loop=(1, 3, 3)),
    # sizes that fit the tensor-core tiles and the split-K products; the loop ends the model
    "tiles": config([
        (attention(8, 2, 32, 16, 40, 32, base=500.0, factor=2.0), moe(64, 8, 2, 4, 2, shared=128)),
        (pair(left(8, 1, 32, coef=0.5, every=24), 2, 64, 64, cap=15.0), moe(128, 4, 1, 2, 1, scale=3.0)),
        (rglru(128, 2), moe(32, 12, 4, 3, 2, scale=2.5, shared=64)),
    ], width=128, vocab=128, loop=(1, 3, 2)),
    # sizes that are no multiple of four, one tap, one head, one block, groups of one expert, no loop
    "odd": config([
        (pair(left(3, 3, 7, every=5), 1, 9, 15), moe(10, 5, 2)),
        (rglru(21, 7, conv=1), moe(7, 3, 1, 3, 2, scale=0.7, shared=9)),
        (attention(5, 1, 10, 6, 7, 2, conv=1), moe(11, 9, 5, 3, 2)),
        (rglru(13, 1, conv=6), None),
        (attention(2, 2, 6, 11, 0, 6, conv=5), None),
    ], width=42, vocab=61, embed_scale=1.0),
    # a model that is one loop, with a matrix memory of several column parts
    "loop": config([
        (pair(left(2, 2, 24, every=32), 1, 72, 330, cap=4.0), moe(24, 4, 2, 2, 2)),
        (attention(4, 4, 24, 24, 32, 16), moe(24, 4, 4)),
    ], width=56, vocab=75, loop=(0, 2, 2)),
}
