"""Palulorn: a pre-norm decoder-only model whose layers are listed in its config.json, some of them run several times.

    x          = "embedding.scale" * embed[tok]                                              (fp32 residual)
    "loop"     : layers start .. stop - 1 run `times` times with the same weights and a cache and state of their own each
                 time; ahead of pass t  x <- W_in [x ; x_0] + step_t, x_0 the embedding's result (layers.LoopInput)
    per layer  : x <- x + mixer(norm(x, norm1)) ; x <- x + ff(norm(x, norm2)) (unless "mlp" is null) ;
                 norm(z, w) = z / sqrt(mean(z^2) + eps) * w
    mixer      : "parallel": (norm(left, "left.out") + norm(right, "right.out")) / 2
                 (layers.ParallelMixer + layers.BranchNormResidual)
                 left  — layers.SharedKVAttention: values are keys, query temperature, learned sink, one output gate per
                         head, no rotary turn
                 right — layers.MatrixMemoryMixer: exponential input and forget gates under a cap, running maximum
                 "rglru": layers.RealGatedMixer
                 "attention": layers.FilteredWindowAttention: short filters on q, k, v, per-head norms, half-pair turn with
                 linearly scaled frequencies, sliding window
    feed-forward: "moe" (layers.GroupSigmoidMoE: squared-ReLU experts, group-limited sigmoid router, shared expert)
    output     : norm(x, "final.norm"), then the vocabulary projection.

Every size and constant is read from config.json or a tensor's shape.  Tensor names: "embed", "head", "final.norm",
"loop.in|step", and per layer i "l<i>.norm1|norm2", "l<i>.mix.left.q|k|o (.b)|g|sink|out",
"l<i>.mix.right.q|k|v|g|o|norm|i|f (.b)|out" (parallel), "l<i>.mix.y|x|conv|ra|ri (.b)|lam|o" (rglru),
"l<i>.mix.q|k|v (.b, .conv)|q.norm|k.norm|o" (attention), "l<i>.mlp.router", "l<i>.mlp.e<j>|shared.up|down".

State per sequence and run of a layer: keys (and values) in paged KVCache rows; matrices, recurrent rows and the filters'
last inputs in state slots.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional, Tuple

import torch

from . import _lib, kernels
from .layers import (BranchNormResidual, FilteredWindowAttention, GroupSigmoidMoE, InputParameters, KVCache, Linear,
                     LoopInput, MatrixMemoryMixer, ParallelMixer, PreNormInput, RealGatedMixer, ReluSquaredMLP,
                     SharedKVAttention, input_rows_multiple)
from .registry import register_model

# constants the design fixes
DECAY_RATE = -8.0            # log a = -8 r softplus(lam)
GROUP_BEST = 2               # a group of experts scores the sum of its two largest
ROUTE_WEIGHT_EPS = 1e-20     # added to the sum of the chosen experts' scores


def rotary_table(rot: Optional[dict]):
    """(frequencies [dims / 2] or None, dims) of a "rot" entry: base^(-2 t / dims), divided by "scaling.factor" where there
    is one; evaluated in float64 and rounded once."""
    if not rot or not int(rot.get("dims") or 0):
        return None, 0
    dims = int(rot["dims"])
    t = torch.arange(dims // 2, dtype=torch.float64)
    f = torch.pow(torch.tensor(float(rot["base"]), dtype=torch.float64), -2.0 * t / dims)
    return (f / float((rot.get("scaling") or {}).get("factor", 1.0))).to(torch.float32), dims


def _attn_sizes(m: dict):
    H, dim = int(m["heads"]), int(m["dim"])
    return H, int(m.get("kv_heads") or H), dim, int(m.get("vdim") or dim)


def layer_runs(config: dict) -> List[Tuple[int, int]]:
    """(layer, pass that starts with this run or -1) in running order."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, -1) for i in range(n)]
    start, stop, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    if not 0 <= start < stop <= n or times < 1:
        raise ValueError(f"loop over layers {start} .. {stop - 1}, {times} times, of {n} layers")
    passes = [(i, t if i == start else -1) for t in range(times) for i in range(start, stop)]
    return [(i, -1) for i in range(start)] + passes + [(i, -1) for i in range(stop, n)]


def tensor_shapes(config: dict) -> Dict[str, tuple]:
    """Names and shapes of a checkpoint of this config."""
    W, V = int(config["width"]), int(config["vocab"])
    out = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
    if config.get("loop"):
        out.update({"loop.in": (W, 2 * W), "loop.step": (int(config["loop"]["times"]), W)})
    for i, L in enumerate(config["layers"]):
        p, m = f"l{i}.", L["mixer"]
        a = p + "mix."
        out[p + "norm1"] = (W,)
        if L["type"] == "parallel":
            H, G, dim, vd = _attn_sizes(m["left"])
            if vd != dim:
                raise ValueError(f"layer {i}: the values are the keys, but a value has {vd} channels and a key {dim}")
            q = a + "left."
            out.update({q + "q": (H * dim, W), q + "q.b": (H * dim,), q + "k": (G * dim, W), q + "k.b": (G * dim,),
                        q + "sink": (H,), q + "g": (H, W), q + "o": (W, H * dim), q + "o.b": (W,), q + "out": (W,)})
            H, dim, vd = (int(m["right"][k]) for k in ("heads", "dim", "vdim"))
            q = a + "right."
            out.update({q + "q": (H * dim, W), q + "k": (H * dim, W), q + "v": (H * vd, W), q + "g": (H * vd, W),
                        q + "o": (W, H * vd), q + "norm": (H * vd,), q + "i": (H, W), q + "i.b": (H,), q + "f": (H, W),
                        q + "f.b": (H,), q + "out": (W,)})
        elif L["type"] == "rglru":
            n, nb = int(m["width"]), int(m["blocks"])
            if n % nb:
                raise ValueError(f"layer {i}: {n} channels do not make {nb} equal blocks")
            out.update({a + "y": (n, W), a + "y.b": (n,), a + "x": (n, W), a + "x.b": (n,), a + "conv": (n, int(m["conv"])),
                        a + "conv.b": (n,), a + "ra": (nb, n // nb, n // nb), a + "ra.b": (nb, n // nb),
                        a + "ri": (nb, n // nb, n // nb), a + "ri.b": (nb, n // nb), a + "lam": (n,), a + "o": (W, n)})
        elif L["type"] == "attention":
            H, G, dim, vd = _attn_sizes(m)
            for name, n in (("q", H * dim), ("k", G * dim), ("v", G * vd)):
                out.update({a + name: (n, W), a + name + ".b": (n,), a + name + ".conv": (n, int(m["conv"]))})
            out.update({a + "q.norm": (dim,), a + "k.norm": (dim,), a + "o": (W, H * vd)})
        else:
            raise ValueError(f"unknown mixer type {L['type']!r}")
        mlp = L.get("mlp")
        if mlp is not None:
            if mlp["kind"] != "moe":
                raise ValueError(f"unknown feed-forward kind {mlp['kind']!r}")
            ff, E, f = int(mlp["expert"]["ff"]), int(mlp["router"]["experts"]), p + "mlp."
            out.update({p + "norm2": (W,), f + "router": (E, W)})
            for e in range(E):
                out.update({f + f"e{e}.up": (ff, W), f + f"e{e}.down": (W, ff)})
            if mlp.get("shared"):
                sf = int(mlp["shared"]["ff"])
                out.update({f + "shared.up": (sf, W), f + "shared.down": (W, sf)})
    return out


def random_tensors(config: dict, seed: int = 0, dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    """Random weights of the architecture (bench and tests): projections N(0, 1/in), gains around one, small biases, decay
    parameters and forget gates in the range where the states forget over tens to hundreds of tokens."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(config).items():
        leaf = name.split(".")[-1]
        if leaf in ("norm1", "norm2", "norm", "out"):
            t = 1.0 + 0.2 * torch.randn(shape, generator=g)
        elif leaf == "lam":
            a = 0.9 + 0.099 * torch.rand(shape, generator=g)           # a = exp(-8 softplus(lam)) at r = 1
            t = torch.log(torch.expm1(-torch.log(a) / 8.0))
        elif name.endswith("right.f.b"):
            t = 3.0 + 2.0 * torch.rand(shape, generator=g)
        elif leaf == "conv":
            t = torch.randn(shape, generator=g) / math.sqrt(shape[-1])
        elif name == "embed":
            t = torch.randn(shape, generator=g) / math.sqrt(shape[-1])
        elif len(shape) == 1 or leaf in ("b", "step"):
            t = 0.2 * torch.randn(shape, generator=g)
        else:
            t = torch.randn(shape, generator=g) / math.sqrt(shape[-1])
        out[name] = t.to(dtype)
    return out


class _Layer:
    read: PreNormInput                        # residual sum and norm1: what the mixer reads
    mixer = None                              # ParallelMixer, RealGatedMixer or FilteredWindowAttention
    join: Optional[BranchNormResidual] = None     # ParallelMixer: how its two results join the residual
    read2: Optional[PreNormInput] = None      # residual sum and norm2: what the feed-forward reads
    ff: Optional[GroupSigmoidMoE] = None


class _Run:
    """One run of a layer: its own cache and state over the layer's weights."""

    def __init__(self, layer: _Layer, step: Optional[torch.Tensor], state):
        self.layer, self.step, self.state = layer, step, state      # step: this run starts a pass
        self.cache: Optional[KVCache] = None


@register_model("Palulorn")
class PalulornDecoder:
    needs_state_slots = True
    CSRC = ("postnorm.cu", "filters.cu", "linear_scan.cu", "mingru.cu", "sink_attn.cu", "moe.cu")

    def __init__(self, config: dict, dtype: torch.dtype, device, max_seqs: int = 4):
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("Palulorn runs in bfloat16 or float32")
        _lib.ensure(self.CSRC)
        self.config, self.dtype, self.device, self.max_seqs = config, dtype, torch.device(device), max_seqs
        self.width, self.n_vocab = int(config["width"]), int(config["vocab"])
        self.eps = float(config["norm"]["eps"])
        self.embed_scale = float((config.get("embedding") or {}).get("scale", 1.0))
        self.layers: List[_Layer] = []
        self.runs: List[_Run] = []
        self.embed = self.final = self.head = self.loop = None

    @classmethod
    def from_config(cls, config: dict, dtype, device, max_seqs: int = 4) -> "PalulornDecoder":
        return cls(config, dtype, device, max_seqs)

    # ------------------------------------------------------------------ weights
    def init_random(self, seed: int = 0) -> None:
        self.load_weights(random_tensors(self.config, seed))

    def load_weights(self, tensors: Dict[str, torch.Tensor]) -> None:
        dev, dt, eps = self.device, self.dtype, self.eps
        for name, shape in tensor_shapes(self.config).items():
            if name not in tensors:
                raise KeyError(f"checkpoint lacks {name}")
            if tuple(tensors[name].shape) != shape:
                raise ValueError(f"{name} is {tuple(tensors[name].shape)}, the config says {shape}")
        w = lambda name: tensors[name].to(dev).to(dt)
        f32 = lambda name: tensors[name].to(dev).to(torch.float32).contiguous()
        self.embed = w("embed").contiguous()
        self.head = Linear(w("head"))
        self.final = PreNormInput(f32("final.norm"), eps)
        self.loop = LoopInput(tensors["loop.in"].to(dev), dt) if self.config.get("loop") else None
        steps = w("loop.step").contiguous() if self.loop is not None else None
        self.layers = [self._load_layer(i, L, tensors, w, f32) for i, L in enumerate(self.config["layers"])]
        self.runs = []
        for i, first_of in layer_runs(self.config):
            mixer = self.layers[i].mixer
            state = (mixer.right if isinstance(mixer, ParallelMixer) else mixer).new_state(self.max_seqs)
            self.runs.append(_Run(self.layers[i], steps[first_of] if first_of >= 0 else None, state))

    def _load_layer(self, i: int, L: dict, tensors: Dict[str, torch.Tensor], w, f32) -> _Layer:
        dev, dt, eps = self.device, self.dtype, self.eps
        p, m, lay = f"l{i}.", L["mixer"], _Layer()
        sub = lambda pre: {k[len(pre):]: w(k) for k in tensors if k.startswith(pre)}
        lay.read = PreNormInput(f32(p + "norm1"), eps)
        if L["type"] == "parallel":
            ml, mr = m["left"], m["right"]
            H, G, dim, _ = _attn_sizes(ml)
            temp = ml.get("q_temp") or {"coef": 0.0, "every": 0}
            left = SharedKVAttention(sub(p + "mix.left."), H, G, dim, float(ml["scale"]), float(temp["coef"]),
                                     int(temp["every"]), dt, dev)
            right = MatrixMemoryMixer(sub(p + "mix.right."), int(mr["heads"]), int(mr["dim"]), int(mr["vdim"]),
                                      float(mr["gate_cap"]), eps, dt, dev)
            lay.mixer = ParallelMixer(left, right, input_rows_multiple(left.n_in + right.n_in))
            lay.join = BranchNormResidual(None, eps, f32(p + "mix.left.out"), f32(p + "mix.right.out"),
                                          bias_a=f32(p + "mix.left.o.b"))
        elif L["type"] == "rglru":
            lay.mixer = RealGatedMixer(sub(p + "mix."), DECAY_RATE, dt, dev)
        else:
            inv_freq, rot_dims = rotary_table(m.get("rot"))
            lay.mixer = FilteredWindowAttention(sub(p + "mix."), *_attn_sizes(m), float(m["scale"]),
                                                int((m.get("mask") or {}).get("size") or 0), inv_freq, rot_dims, eps, dt,
                                                dev)
        mlp = L.get("mlp")
        if mlp is not None:
            f, r = p + "mlp.", mlp["router"]
            grp = r.get("groups") or {}
            stack = lambda leaf: torch.stack([w(f"{f}e{e}.{leaf}") for e in range(int(r["experts"]))], dim=0)
            shared = ReluSquaredMLP(w(f + "shared.up"), w(f + "shared.down")) if mlp.get("shared") else None
            n_groups = int(grp.get("count") or 1)
            lay.ff = GroupSigmoidMoE(tensors[f + "router"].to(dev), stack("up"), stack("down"), int(r["top"]), n_groups,
                                     int(grp.get("keep") or n_groups), GROUP_BEST, ROUTE_WEIGHT_EPS,
                                     float(r.get("scale", 1.0)), dt, shared)
            lay.read2 = PreNormInput(f32(p + "norm2"), eps)
        return lay

    # ------------------------------------------------------------------ cache
    def alloc_cache(self, n_blocks: int, block_size: int) -> None:
        for run in self.runs:
            mixer = run.layer.mixer
            if isinstance(mixer, ParallelMixer):
                a = mixer.left
                run.cache = KVCache(n_blocks, block_size, a.G, a.dim, self.dtype, self.device, shared=True)
            elif isinstance(mixer, FilteredWindowAttention):
                run.cache = KVCache(n_blocks, block_size, mixer.G, mixer.dim, self.dtype, self.device, value_dim=mixer.vd)

    # ------------------------------------------------------------------ forward
    def forward(self, tokens: torch.Tensor, positions: torch.Tensor, params: InputParameters,
                last_token_idxes: Optional[torch.Tensor] = None, layer_out: Optional[list] = None) -> torch.Tensor:
        """One step over the packed rows of all sequences; logits [rows or len(last_token_idxes), vocab].
        layer_out, if given, receives the residual after every run of a layer (fp32).  A sublayer's result y joins the
        residual in the launch that makes the next sublayer's input."""
        dt = self.dtype
        x, _ = kernels.bigram_embed(self.embed, None, tokens, None, 0, 0, 0, self.embed_scale, want_h=False)
        both = self.loop.start(x) if self.loop is not None else None
        y = None
        for n, run in enumerate(self.runs):
            lay = run.layer
            if run.step is not None:
                x, start = self.loop(x, y, both)
                ended = x
                x, h = lay.read(start, run.step, dt, positions, params)
            else:
                x, h = lay.read(x, y, dt, positions, params)
                ended = x
            if layer_out is not None and n > 0:
                layer_out.append(ended.clone())
            if lay.join is not None:
                a, b = lay.mixer(h, positions, run.cache, params, h, run.state)
                ff = lay.ff is not None
                x, h = lay.join(x, a, b, next_weight=lay.read2.weight if ff else None, want_h=ff)
                y = lay.ff(h) if ff else None
                continue
            if run.cache is not None:
                y = lay.mixer(h, positions, run.cache, params, run.state)
            else:
                y = lay.mixer(h, positions, params, run.state)
            if lay.ff is not None:
                x, h = lay.read2(x, y, dt, positions, params)
                y = lay.ff(h)
        rows = None if last_token_idxes is None else last_token_idxes.to(torch.int64)
        few = rows is not None and 2 * rows.numel() <= x.shape[0]       # the last norm runs over the asked rows only
        if few and layer_out is None and (y is None or isinstance(y, torch.Tensor)):
            x, y, rows = x.index_select(0, rows), None if y is None else y.index_select(0, rows), None
        x, h = self.final(x, y, dt, positions, params)
        if layer_out is not None:
            layer_out.append(x.clone())
        return self.head(h if rows is None else h.index_select(0, rows))

    __call__ = forward
