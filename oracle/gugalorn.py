"""oracle.gugalorn — the Gugalorn decoder restated in plain torch on the CPU.  TEST INFRASTRUCTURE.

One function per mechanism, written from the design's equations and sharing nothing with the
product path (`scalellm_b200/`).  Everything runs in one floating-point type (float64 by default)
over an explicit per-sequence state, so the same functions serve whole prompts, portions and
single decoded tokens.

Notation (W = width, norm(x, w) = x / sqrt(mean(x^2) + eps) * w):

    x_0         = s_e * embed[tok]
    layer       : h = norm(x, n1) ; h <- h + filter(h) ; x <- x + mixer(h) ; x <- x + ff(norm(x, n2))  (no ff: skipped)
    filter      : y_t = sum_j c[:, j] h_{t - (taps - 1) + j} per channel, zeros before the start of the sequence
    "mamba2"    : [z | x | B | C | dt] = Win h ; [x | B | C] <- silu(filter(.) + b) ; dt <- softplus(dt + dt_bias) ;
                  per head (N x vdim state, group of head h: h // (heads / groups)):
                  S <- exp(-exp(A_log) dt) S + dt B x^T ; y = S^T C + D x ;
                  y <- y * silu(z), each of norm_groups equal parts over its root mean square, times w ; result Wo y
    "parallel"  : s_l left(h) + s_r right(h)
    left        : q, k, v, g = Wq h, Wk h, Wv h, Wg h ; q, k <- norm over ALL rows of the projection ; the first rot.dims
                  channels of every head turn (channel i with i + dims / 2, angle p base^(-2 i / dims)) ;
                  s_ij = scale q_i . k_j for j <= i ; p_ij = exp(s_ij) / (1 + sum_j exp(s_ij)) ;
                  result Wo (concat_h(sum_j p_ij v_j) * sigmoid(g))
    right       : q = silu(Wq h), f = l + (1 - l) sigmoid(Wf h + b), v = Wv h ; per head
                  S <- diag(f) S + (1 - f) v^T ; o = S^T q ; result Wo concat_h(norm(o, w))
    ff "dense"  : Wd (silu(Wg h) * (Wu h))
    output      : embed norm(x, final)      (tied weights)
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from .kigalix import read_safetensors  # noqa: F401  (same file format)


def norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def filter_causal(x: torch.Tensor, c: torch.Tensor, st: Dict[str, torch.Tensor], key: str) -> torch.Tensor:
    """x [T, channels] new inputs, c [channels, taps]; st[key] keeps the last taps - 1 inputs of the sequence."""
    taps = c.shape[1]
    if key not in st:
        st[key] = torch.zeros(taps - 1, x.shape[1], dtype=x.dtype)
    ext = torch.cat([st[key], x], dim=0)
    y = torch.zeros_like(x)
    for j in range(taps):
        y = y + c[:, j] * ext[j: j + x.shape[0]]
    st[key] = ext[ext.shape[0] - (taps - 1):].clone()
    return y


# ------------------------------------------------------------------------------------------------ mamba2
def ssd_scan(x: torch.Tensor, B: torch.Tensor, C: torch.Tensor, dt: torch.Tensor, a_log: torch.Tensor,
             D: torch.Tensor, S: torch.Tensor) -> torch.Tensor:
    """x [T, heads, vdim], B, C [T, groups, N], dt [T, heads] (after softplus); S [heads, N, vdim] is carried."""
    T, H, G = x.shape[0], x.shape[1], B.shape[1]
    y = torch.zeros_like(x)
    for t in range(T):
        for h in range(H):
            g = h // (H // G)
            S[h] = torch.exp(-torch.exp(a_log[h]) * dt[t, h]) * S[h] + dt[t, h] * torch.outer(B[t, g], x[t, h])
            y[t, h] = S[h].T @ C[t, g] + D[h] * x[t, h]
    return y


def gated_part_norm(y: torch.Tensor, z: torch.Tensor, w: torch.Tensor, parts: int, eps: float) -> torch.Tensor:
    """The gate first, then every part of the row over its own root mean square."""
    u = y * silu(z)
    T, n = u.shape
    p = u.reshape(T, parts, n // parts)
    p = p / torch.sqrt((p * p).mean(dim=-1, keepdim=True) + eps)
    return p.reshape(T, n) * w


def mamba2_mixer(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float, st: Dict) -> torch.Tensor:
    H, vd, N, G = int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m["groups"])
    T, inner = h.shape[0], H * vd
    p = h @ w["in"].T
    z, xbc, dt = p[:, :inner], p[:, inner: 2 * inner + 2 * G * N], p[:, 2 * inner + 2 * G * N:]
    xbc = silu(filter_causal(xbc, w["conv"], st, "conv") + w["conv.b"])
    x = xbc[:, :inner].reshape(T, H, vd)
    B = xbc[:, inner: inner + G * N].reshape(T, G, N)
    C = xbc[:, inner + G * N:].reshape(T, G, N)
    dt = torch.log1p(torch.exp(-torch.abs(dt + w["dt_bias"]))) + torch.clamp(dt + w["dt_bias"], min=0.0)
    if "S" not in st:
        st["S"] = torch.zeros(H, N, vd, dtype=h.dtype)
    y = ssd_scan(x, B, C, dt, w["A_log"], w["D"], st["S"]).reshape(T, inner)
    return gated_part_norm(y, z, w["norm"], int(m["norm_groups"]), eps) @ w["o"].T


# ------------------------------------------------------------------------------------------------ left half
def turn(x: torch.Tensor, pos: torch.Tensor, base: float, dims: int) -> torch.Tensor:
    """x [T, heads, n]: the first `dims` channels of every head turn, channel i with channel i + dims / 2."""
    half = dims // 2
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float64)
    a = pos.to(torch.float64)[:, None] * f[None, :]
    c, s = torch.cos(a).to(x.dtype)[:, None, :], torch.sin(a).to(x.dtype)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def attend_with_one(q: torch.Tensor, K: torch.Tensor, V: torch.Tensor, pos: torch.Tensor, scale: float) -> torch.Tensor:
    """q [T, H, dim] at positions pos over keys K [n, G, dim] and values V [n, G, vd] of positions 0 .. n - 1: causal
    softmax whose denominator has one more term, exp(0) = 1."""
    T, H, G = q.shape[0], q.shape[1], K.shape[1]
    out = torch.zeros(T, H, V.shape[2], dtype=q.dtype)
    j = torch.arange(K.shape[0])
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ K[:, g].T) * scale
        s = torch.where(j[None, :] <= pos[:, None], s, torch.full_like(s, -torch.inf))
        top = torch.clamp(s.max(dim=1, keepdim=True).values, min=0.0)
        e = torch.exp(s - top)
        out[:, h] = (e / (torch.exp(-top) + e.sum(dim=1, keepdim=True))) @ V[:, g]
    return out


def left_half(h: torch.Tensor, pos: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float,
              st: Dict) -> torch.Tensor:
    H, G, dim, vd = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    T = h.shape[0]
    q = norm(h @ w["q"].T, w["q.norm"], eps).reshape(T, H, dim)
    k = norm(h @ w["k"].T, w["k.norm"], eps).reshape(T, G, dim)
    v = (h @ w["v"].T).reshape(T, G, vd)
    base, dims = float(m["rot"]["base"]), int(m["rot"]["dims"])
    q, k = turn(q, pos, base, dims), turn(k, pos, base, dims)
    st["K"] = torch.cat([st["K"], k]) if "K" in st else k
    st["V"] = torch.cat([st["V"], v]) if "V" in st else v
    o = attend_with_one(q, st["K"], st["V"], pos, float(m["scale"])).reshape(T, H * vd)
    return (o * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


# ------------------------------------------------------------------------------------------------ right half
def forget_write_scan(q: torch.Tensor, f: torch.Tensor, v: torch.Tensor, S: torch.Tensor) -> torch.Tensor:
    """q, f [T, H, dim], v [T, H, vd]; S [H, dim, vd] is carried: what a channel forgets it writes anew."""
    o = torch.zeros_like(v)
    for t in range(q.shape[0]):
        S.copy_(f[t][:, :, None] * S + (1.0 - f[t])[:, :, None] * v[t][:, None, :])
        o[t] = (S * q[t][:, :, None]).sum(dim=1)
    return o


def right_half(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float, st: Dict) -> torch.Tensor:
    H, dim, vd = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    T = h.shape[0]
    q = silu(h @ w["q"].T).reshape(T, H, dim)
    low = w["lower"]
    f = (low + (1.0 - low) * torch.sigmoid(h @ w["f"].T + w["f.b"])).reshape(T, H, dim)
    v = (h @ w["v"].T).reshape(T, H, vd)
    if "S" not in st:
        st["S"] = torch.zeros(H, dim, vd, dtype=h.dtype)
    o = norm(forget_write_scan(q, f, v, st["S"]), w["norm"], eps)
    return o.reshape(T, H * vd) @ w["o"].T


def parallel_mixer(h, pos, w, m, eps, st) -> torch.Tensor:
    sub = lambda p: {k[len(p):]: v for k, v in w.items() if k.startswith(p)}
    a = left_half(h, pos, sub("left."), m["left"], eps, st.setdefault("left", {}))
    b = right_half(h, sub("right."), m["right"], eps, st.setdefault("right", {}))
    return float(m["left_scale"]) * a + float(m["right_scale"]) * b


def dense_ff(h: torch.Tensor, w: Dict[str, torch.Tensor]) -> torch.Tensor:
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


# ------------------------------------------------------------------------------------------------ the model
class Gugalorn:
    def __init__(self, config: dict, tensors: Dict[str, torch.Tensor], dtype=torch.float64):
        self.cfg, self.dtype = config, dtype
        self.w = {k: v.to(dtype) for k, v in tensors.items()}
        self.eps = float(config["norm"]["eps"])

    def new_state(self) -> dict:
        return {"pos": 0, "layers": [{} for _ in self.cfg["layers"]]}

    def forward(self, tokens: List[int], state: dict, layer_out: Optional[list] = None) -> torch.Tensor:
        """Logits of every given token; `state` moves on."""
        W, eps = self.w, self.eps
        pos = torch.arange(state["pos"], state["pos"] + len(tokens))
        x = W["embed"][torch.tensor(tokens)] * float(self.cfg["embedding"]["scale"])
        for i, L in enumerate(self.cfg["layers"]):
            st, p = state["layers"][i], f"l{i}."
            sub = lambda pre: {k[len(pre):]: v for k, v in W.items() if k.startswith(pre)}
            h = norm(x, W[p + "norm1"], eps)
            h = h + filter_causal(h, W[p + "canon1"], st, "canon")
            if L["type"] == "mamba2":
                x = x + mamba2_mixer(h, sub(p + "mix."), L["mixer"], eps, st)
            else:
                x = x + parallel_mixer(h, pos, sub(p + "mix."), L["mixer"], eps, st)
            if L["mlp"] is not None:
                x = x + dense_ff(norm(x, W[p + "norm2"], eps), sub(p + "mlp."))
            if layer_out is not None:
                layer_out.append(x.clone())
        state["pos"] += len(tokens)
        return norm(x, W["final.norm"], eps) @ W["embed"].T
