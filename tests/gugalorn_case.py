"""Small Gugalorn configurations and weights for the tests (not the product's generator: shapes are derived here from the
config, so the product's own shape table is checked against this one)."""
import math

import torch


def mamba(heads, vdim, state, groups, parts, conv=4):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups,
                                        "norm_groups": parts, "conv": conv}}


def left(heads, kv_heads, dim, vdim, rot_dims, base=10000.0, scale=None):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
            "scale": scale if scale is not None else 1.0 / math.sqrt(dim), "rot": {"base": base, "dims": rot_dims}}


def right(heads, dim, vdim):
    return {"heads": heads, "dim": dim, "vdim": vdim}


def pair(a, b, left_scale=0.8, right_scale=0.7):
    return {"type": "parallel", "mixer": {"left": a, "right": b, "left_scale": left_scale, "right_scale": right_scale}}


def config(layers, width=64, vocab=97, eps=1e-5, taps=4, embed_scale=2.0):
    """layers: list of (mixer entry, feed-forward width or None)."""
    return {"architecture": "Gugalorn", "width": width, "vocab": vocab, "norm": {"eps": eps}, "canon": {"taps": taps},
            "embedding": {"scale": embed_scale},
            "layers": [dict(m, mlp={"kind": "dense", "ff": ff} if ff else None) for m, ff in layers]}


def shapes(cfg):
    W, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, W), "final.norm": (W,)}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        out[p + "norm1"], out[p + "canon1"] = (W,), (W, cfg["canon"]["taps"])
        if L["type"] == "mamba2":
            H, v, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
            ch = H * v + 2 * G * N
            out.update({p + "mix.in": (H * v + ch + H, W), p + "mix.conv": (ch, m["conv"]), p + "mix.conv.b": (ch,),
                        p + "mix.dt_bias": (H,), p + "mix.A_log": (H,), p + "mix.D": (H,), p + "mix.norm": (H * v,),
                        p + "mix.o": (W, H * v)})
        else:
            a, b = m["left"], m["right"]
            H, G, d, v = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            q = p + "mix.left."
            out.update({q + "q": (H * d, W), q + "k": (G * d, W), q + "v": (G * v, W), q + "q.norm": (H * d,),
                        q + "k.norm": (G * d,), q + "g": (H * v, W), q + "o": (W, H * v)})
            H, d, v = b["heads"], b["dim"], b["vdim"]
            q = p + "mix.right."
            out.update({q + "q": (H * d, W), q + "f": (H * d, W), q + "f.b": (H * d,), q + "lower": (H * d,),
                        q + "v": (H * v, W), q + "norm": (v,), q + "o": (W, H * v)})
        if L["mlp"] is not None:
            ff = L["mlp"]["ff"]
            out[p + "norm2"] = (W,)
            out.update({p + "mlp.gate": (ff, W), p + "mlp.up": (ff, W), p + "mlp.down": (W, ff)})
    return out


def weights(cfg, seed=0):
    """bf16 tensors: projections N(0, 1/in), gains around one; the keys' gains are large so that attention is sharp
    and a wrong key shows; step sizes and lower bounds from nearly forgetful to nearly lossless."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shp in shapes(cfg).items():
        leaf = name.split(".")[-1]
        if name.endswith("left.k.norm"):
            t = 2.5 + 0.5 * torch.randn(shp, generator=g)
        elif leaf in ("norm1", "norm2", "norm", "D"):
            t = 1.0 + 0.3 * torch.randn(shp, generator=g)
        elif leaf == "A_log":
            t = torch.log(0.2 + 4.0 * torch.rand(shp, generator=g))
        elif leaf == "dt_bias":
            t = -4.0 + 4.0 * torch.rand(shp, generator=g)
        elif leaf in ("conv", "canon1"):
            t = 0.5 * torch.randn(shp, generator=g)
        elif leaf == "lower":
            t = torch.rand(shp, generator=g) ** 0.5 * 0.98
        elif name == "embed":
            t = torch.randn(shp, generator=g) / math.sqrt(shp[-1]) * 2.0
        elif len(shp) == 1:
            t = 0.5 * torch.randn(shp, generator=g)
        else:
            t = torch.randn(shp, generator=g) / math.sqrt(shp[-1])
        out[name] = t.to(torch.bfloat16)
    return out


def row_errors(got, want):
    """Per row: root mean square of the difference of the mean-free logits over that of the wanted ones."""
    got, want = got.double().cpu(), want.double().cpu()
    got = got - got.mean(dim=-1, keepdim=True)
    want = want - want.mean(dim=-1, keepdim=True)
    return (got - want).pow(2).mean(dim=-1).sqrt() / want.pow(2).mean(dim=-1).sqrt()


CONFIGS = {
    # sizes that differ from each other on every side, both mixers with and without a feed-forward, norm parts that cut
    # through heads
    "mix": config([
        (mamba(6, 10, 24, 3, 4, conv=4), 40),
        (pair(left(4, 2, 16, 24, 8), right(3, 20, 12), 0.8, 0.3), None),
        (pair(left(6, 2, 12, 20, 12, base=100.0), right(2, 40, 36), 0.4, 1.1), 96),
        (mamba(2, 36, 8, 1, 1, conv=2), None),
    ], taps=3),
    # sizes that fit the tensor-core tiles and the split-K products
    "tiles": config([
        (mamba(4, 32, 64, 2, 2, conv=4), None),
        (pair(left(8, 2, 32, 16, 16), right(2, 64, 64), 0.9, 0.6), 128),
        (mamba(2, 64, 128, 1, 2, conv=3), 256),
        (pair(left(4, 1, 16, 32, 4, scale=0.4), right(4, 32, 32), 1.0, 1.0), 128),
    ], width=128, vocab=128, taps=4),
    # sizes that are no multiple of four, one tap, one head, groups of one head
    "odd": config([
        (mamba(5, 6, 7, 5, 3, conv=1), 30),
        (pair(left(3, 3, 10, 7, 2), right(1, 9, 15), 1.3, 0.5), 22),
        (mamba(1, 13, 18, 1, 1, conv=5), None),
        (pair(left(5, 1, 6, 5, 6), right(5, 6, 11), 0.7, 0.7), None),
    ], width=42, vocab=61, taps=1, embed_scale=1.0),
    # more taps than most portions have tokens, key and value sizes of several column and row parts
    "wide": config([
        (pair(left(2, 1, 64, 72, 64), right(1, 150, 136), 0.5, 0.5), 48),
        (mamba(2, 140, 130, 2, 4, conv=6), 32),
    ], width=48, vocab=70, taps=6),
}
