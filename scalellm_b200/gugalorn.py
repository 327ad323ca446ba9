"""Gugalorn: a pre-norm decoder-only model whose layers are listed in its config.json.

    x          = "embedding.scale" * embed[tok]                                              (fp32 residual)
    per layer  : h = norm(x, norm1) ; h_t <- h_t + sum_i canon1[:, i] h_{t - (taps - 1) + i}   (layers.PreNormInput) ;
                 x <- x + mixer(h) ; x <- x + ff(norm(x, norm2)) (unless "mlp" is null) ;
                 norm(z, w) = z / sqrt(mean(z^2) + eps) * w
    mixer      : "mamba2"   layers.StateSpaceMixer
                 "parallel" layers.ScaledPairMixer of
                 left  — layers.TurnedSinkAttention: norms over the whole query / key projection, partial rotary turn over
                         channel pairs (t, t + dims / 2), grouped key/value heads, softmax with a sink of score 0, output
                         gate
                 right — layers.ForgetWriteMixer: forget gate with a lower bound per channel, per-head norm of the read-out
    feed-forward: "dense" (layers.GatedMLP with silu)
    output     : norm(x, "final.norm"), then the vocabulary projection with the weights of embed.

Every size and constant is read from config.json or a tensor's shape.  Tensor names: "embed", "final.norm", and per
layer i "l<i>.norm1|norm2|canon1", "l<i>.mix.in|conv|conv.b|dt_bias|A_log|D|norm|o" (mamba2),
"l<i>.mix.left.q|k|v|q.norm|k.norm|g|o" and "l<i>.mix.right.q|f|f.b|lower|v|norm|o" (parallel), "l<i>.mlp.gate|up|down".

State per sequence: the turned keys and the values of the left halves in paged KVCache rows; in state slots the last
inputs of every layer's input filter, the state matrices of both recurrences and the last inputs of the state-space
mixer's own filter.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

from . import _lib, kernels
from .layers import (ForgetWriteMixer, GatedMLP, InputParameters, KVCache, Linear, PreNormInput, ScaledPairMixer,
                     StateSpaceMixer, TurnedSinkAttention)
from .registry import register_model

SINK_SCORE = 0.0             # the design's sink: exp(0) = 1 joins the softmax denominator


def rotary_frequencies(base: float, dims: int) -> torch.Tensor:
    """base^(-2 t / dims) for t < dims / 2, evaluated in float64 and rounded once."""
    t = torch.arange(dims // 2, dtype=torch.float64)
    return torch.pow(torch.tensor(base, dtype=torch.float64), -2.0 * t / dims).to(torch.float32)


def _left_sizes(m: dict):
    return int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])


def _right_sizes(m: dict):
    return int(m["heads"]), int(m["dim"]), int(m["vdim"])


def tensor_shapes(config: dict) -> Dict[str, tuple]:
    """Names and shapes of a checkpoint of this config."""
    W, V, taps = int(config["width"]), int(config["vocab"]), int(config["canon"]["taps"])
    out = {"embed": (V, W), "final.norm": (W,)}
    for i, L in enumerate(config["layers"]):
        p, m = f"l{i}.", L["mixer"]
        out[p + "norm1"] = (W,)
        out[p + "canon1"] = (W, taps)
        a = p + "mix."
        if L["type"] == "mamba2":
            H, vd, N, G = int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m["groups"])
            inner, ch = H * vd, H * vd + 2 * G * N
            out.update({a + "in": (inner + ch + H, W), a + "conv": (ch, int(m["conv"])), a + "conv.b": (ch,),
                        a + "dt_bias": (H,), a + "A_log": (H,), a + "D": (H,), a + "norm": (inner,),
                        a + "o": (W, inner)})
        elif L["type"] == "parallel":
            H, G, dim, vd = _left_sizes(m["left"])
            out.update({a + "left.q": (H * dim, W), a + "left.k": (G * dim, W), a + "left.v": (G * vd, W),
                        a + "left.q.norm": (H * dim,), a + "left.k.norm": (G * dim,), a + "left.g": (H * vd, W),
                        a + "left.o": (W, H * vd)})
            H, dim, vd = _right_sizes(m["right"])
            out.update({a + "right.q": (H * dim, W), a + "right.f": (H * dim, W), a + "right.f.b": (H * dim,),
                        a + "right.lower": (H * dim,), a + "right.v": (H * vd, W), a + "right.norm": (vd,),
                        a + "right.o": (W, H * vd)})
        else:
            raise ValueError(f"unknown mixer type {L['type']!r}")
        mlp = L.get("mlp")
        if mlp is not None:
            if mlp["kind"] != "dense":
                raise ValueError(f"unknown feed-forward kind {mlp['kind']!r}")
            ff = int(mlp["ff"])
            out[p + "norm2"] = (W,)
            out.update({p + "mlp.gate": (ff, W), p + "mlp.up": (ff, W), p + "mlp.down": (W, ff)})
    return out


def random_tensors(config: dict, seed: int = 0, dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    """Random weights of the architecture (bench and tests): projections N(0, 1/in), gains around one, small biases,
    step sizes and forget gates in the range where the states forget over tens to thousands of tokens."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(config).items():
        leaf = name.split(".")[-1]
        if leaf in ("norm1", "norm2", "norm", "D"):
            t = 1.0 + 0.2 * torch.randn(shape, generator=g)
        elif leaf == "A_log":
            t = torch.log(1.0 + 15.0 * torch.rand(shape, generator=g))
        elif leaf == "dt_bias":
            dt = torch.exp(math.log(1e-3) + (math.log(1e-1) - math.log(1e-3)) * torch.rand(shape, generator=g))
            t = dt + torch.log(-torch.expm1(-dt))                  # softplus(t) = dt
        elif leaf in ("conv", "canon1"):
            t = torch.randn(shape, generator=g) / shape[-1]
        elif leaf == "lower":
            t = 0.99 * torch.rand(shape, generator=g)
        elif name == "embed":
            t = torch.randn(shape, generator=g) / math.sqrt(shape[-1])
        elif len(shape) == 1:
            t = 0.2 * torch.randn(shape, generator=g)
        else:
            t = torch.randn(shape, generator=g) / math.sqrt(shape[-1])
        out[name] = t.to(dtype)
    return out


class _Layer:
    read: PreNormInput                        # residual sum, norm1 and input filter: what the mixer reads
    mixer = None                              # StateSpaceMixer or ScaledPairMixer
    read2: Optional[PreNormInput] = None      # residual sum and norm2: what the feed-forward reads
    ff: Optional[GatedMLP] = None
    cache: Optional[KVCache] = None           # layers with an attention half


@register_model("Gugalorn")
class GugalornDecoder:
    needs_state_slots = True
    CSRC = ("postnorm.cu", "hyper.cu", "filters.cu", "linear_scan.cu", "sink_attn.cu")

    def __init__(self, config: dict, dtype: torch.dtype, device, max_seqs: int = 4):
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("Gugalorn runs in bfloat16 or float32")
        _lib.ensure(self.CSRC)
        self.config, self.dtype, self.device, self.max_seqs = config, dtype, torch.device(device), max_seqs
        self.width, self.n_vocab = int(config["width"]), int(config["vocab"])
        self.eps = float(config["norm"]["eps"])
        self.embed_scale = float(config["embedding"]["scale"])
        self.layers: List[_Layer] = []
        self.embed = self.final = self.head = None

    @classmethod
    def from_config(cls, config: dict, dtype, device, max_seqs: int = 4) -> "GugalornDecoder":
        return cls(config, dtype, device, max_seqs)

    # ------------------------------------------------------------------ weights
    def init_random(self, seed: int = 0) -> None:
        self.load_weights(random_tensors(self.config, seed))

    def load_weights(self, tensors: Dict[str, torch.Tensor]) -> None:
        dev, dt, eps, n_slots = self.device, self.dtype, self.eps, self.max_seqs
        for name, shape in tensor_shapes(self.config).items():
            if name not in tensors:
                raise KeyError(f"checkpoint lacks {name}")
            if tuple(tensors[name].shape) != shape:
                raise ValueError(f"{name} is {tuple(tensors[name].shape)}, the config says {shape}")
        w = lambda name: tensors[name].to(dev).to(dt)
        f32 = lambda name: tensors[name].to(dev).to(torch.float32).contiguous()
        self.embed = w("embed").contiguous()
        self.head = Linear(self.embed)
        self.final = PreNormInput(f32("final.norm"), eps)
        self.layers = []
        for i, L in enumerate(self.config["layers"]):
            p, m, lay = f"l{i}.", L["mixer"], _Layer()
            sub = lambda pre: {k[len(pre):]: w(k) for k in tensors if k.startswith(pre)}
            lay.read = PreNormInput(f32(p + "norm1"), eps, f32(p + "canon1"), n_slots)
            if L["type"] == "mamba2":
                lay.mixer = StateSpaceMixer(sub(p + "mix."), int(m["heads"]), int(m["vdim"]), int(m["state"]),
                                            int(m["groups"]), int(m["norm_groups"]), eps, n_slots, dt, dev)
            else:
                ml = m["left"]
                rot_dims = int(ml["rot"]["dims"])
                inv_freq = rotary_frequencies(float(ml["rot"]["base"]), rot_dims) if rot_dims else None
                left = TurnedSinkAttention(sub(p + "mix.left."), *_left_sizes(ml), float(ml["scale"]), SINK_SCORE,
                                           inv_freq, rot_dims, eps, dt, dev)
                right = ForgetWriteMixer(sub(p + "mix.right."), *_right_sizes(m["right"]), eps, n_slots, dt, dev)
                lay.mixer = ScaledPairMixer(left, right, float(m["left_scale"]), float(m["right_scale"]))
            if L.get("mlp") is not None:
                f = p + "mlp."
                lay.ff = GatedMLP(w(f + "gate"), w(f + "up"), w(f + "down"), "silu")
                lay.read2 = PreNormInput(f32(p + "norm2"), eps)
            self.layers.append(lay)

    # ------------------------------------------------------------------ cache
    def alloc_cache(self, n_blocks: int, block_size: int) -> None:
        for lay, L in zip(self.layers, self.config["layers"]):
            if L["type"] == "parallel":
                _, G, dim, vd = _left_sizes(L["mixer"]["left"])
                lay.cache = KVCache(n_blocks, block_size, G, dim, self.dtype, self.device, value_dim=vd)

    # ------------------------------------------------------------------ forward
    def forward(self, tokens: torch.Tensor, positions: torch.Tensor, params: InputParameters,
                last_token_idxes: Optional[torch.Tensor] = None, layer_out: Optional[list] = None) -> torch.Tensor:
        """One step over the packed rows of all sequences; logits [rows or len(last_token_idxes), vocab].
        layer_out, if given, receives the residual after every layer (fp32).  Every sublayer's result y joins the
        residual in the launch that makes the next sublayer's input."""
        dt = self.dtype
        x, _ = kernels.bigram_embed(self.embed, None, tokens, None, 0, 0, 0, self.embed_scale, want_h=False)
        y = None
        for i, lay in enumerate(self.layers):
            x, h = lay.read(x, y, dt, positions, params)
            if layer_out is not None and i > 0:
                layer_out.append(x.clone())
            y = (lay.mixer(h, positions, params) if isinstance(lay.mixer, StateSpaceMixer)
                 else lay.mixer(h, positions, lay.cache, params))
            if lay.ff is not None:
                x, h = lay.read2(x, y, dt, positions, params)
                y = lay.ff(h, fusable_out=True)
        x, h = self.final(x, y, dt, positions, params)
        if layer_out is not None:
            layer_out.append(x.clone())
        if last_token_idxes is not None:
            h = h.index_select(0, last_token_idxes.to(torch.int64))
        return self.head(h)

    __call__ = forward
