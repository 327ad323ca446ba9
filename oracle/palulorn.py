"""oracle.palulorn — the Palulorn decoder restated in plain torch on the CPU.  TEST INFRASTRUCTURE.

One function per mechanism, written from the design's equations and sharing nothing with the
product path (`scalellm_b200/`).  Everything runs in one floating-point type (float64 by default)
over an explicit per-sequence state, so the same functions serve whole prompts, portions and
single decoded tokens.

Notation (norm(x, w) = x / sqrt(mean(x^2) + eps) * w; b_*: biases):

    x_0         = s_e * embed[tok]
    loop        : layers start .. stop - 1 run `times` times; ahead of pass t  x <- W_in [x ; x_0] + step_t
    layer       : x <- x + mixer(norm(x, n1)) ; x <- x + ff(norm(x, n2))  (no ff: skipped)
    "parallel"  : (norm(left(h), w_l) + norm(right(h), w_r)) / 2
    left        : q = Wq h + b_q, k = v = Wk h + b_k ; q <- q (1 + c ln(floor((p + 1) / n) + 1)) at position p ;
                  s_ij = scale q_i . k_j, j <= i ; p_ij = exp(s_ij) / (exp(sink) + sum_j exp(s_ij)) ;
                  Wo concat_h(sum_j p_ij k_j * sigmoid(Wg h)_h) + b_o
    right       : q = Wq h / sqrt(dim), k = Wk h, v = Wv h ; i = cap tanh((Wi h + b_i) / cap) ,
                  f = log sigmoid(cap tanh((Wf h + b_f) / cap)) ; m_t = max(f + m, i) from m = 0 ;
                  (S, n) <- exp(f + m - m_t) (S, n) + exp(i - m_t) k (v^T, 1) ;
                  o = S^T q / (max(|n . q|, exp(-m_t)) + 1e-6) ; Wo (norm_head(o) * w * sigmoid(Wg h))
    "rglru"     : y = gelu_tanh(Wy h + b_y) ; u = filter(Wx h + b_x) + b_c ; per block r, i = sigmoid(R u + b), sigmoid(I u + b) ;
                  log a = -8 r softplus(lam) ; S <- a S + sqrt(1 - a^2) i u ; Wo (S y)
    "attention" : q, k, v = filter(W h + b) ; per-head norms of q and k ; half-pair turn of the first rot.dims channels,
                  frequencies base^(-2 i / dims) / factor ; softmax of scale q . k over 0 <= i - j < size ; Wo
    ff "moe"    : s = sigmoid(R h) ; groups of neighbours score the sum of their two largest s, the best `keep` stay ;
                  the `top` largest s ; weight = factor s / (sum of the chosen s + 1e-20) ;
                  sum weight * Wd relu(Wu h)^2 (+ the shared expert)
    output      : head norm(x, final)
"""
from __future__ import annotations

import contextlib
import math
from typing import Dict, List, Optional

import torch

from .kigalix import read_safetensors  # noqa: F401  (same file format)


_shake: Optional[torch.Generator] = None


@contextlib.contextmanager
def shaken(seed: int):
    """Inside, the results of norms and of matrix products are off by up to the distance between neighbouring 16-bit
    numbers (2^-8 of their size): what rounding in a 16-bit model may do to a row."""
    global _shake
    _shake = torch.Generator().manual_seed(seed)
    try:
        yield
    finally:
        _shake = None


def stored(x: torch.Tensor) -> torch.Tensor:
    if _shake is None:
        return x
    return x * (1.0 + (2.0 * torch.rand(x.shape, generator=_shake, dtype=x.dtype) - 1.0) * 2.0 ** -8)


def norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return stored(x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w)


def apply(w: torch.Tensor, h: torch.Tensor) -> torch.Tensor:
    """W h for rows h."""
    return stored(h @ w.T)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def log_sigmoid(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, max=0.0) - torch.log1p(torch.exp(-z.abs()))


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def short_filter(x: torch.Tensor, c: torch.Tensor, st: Dict[str, torch.Tensor], key: str) -> torch.Tensor:
    """x [T, channels] new inputs, c [channels, taps] (last column: the current token); st[key]: the last taps - 1."""
    taps = c.shape[1]
    before = st.get(key)
    if before is None:
        before = torch.zeros(taps - 1, x.shape[1], dtype=x.dtype)
    ext = torch.cat([before, x])
    st[key] = ext[x.shape[0]:].clone()
    return sum(c[:, j] * ext[j: j + x.shape[0]] for j in range(taps))


def turn(x: torch.Tensor, pos: torch.Tensor, base: float, dims: int, factor: float) -> torch.Tensor:
    """x [T, heads, n]: channel i < dims / 2 of every head turns with channel i + dims / 2."""
    half = dims // 2
    f = torch.tensor([base ** (-2.0 * i / dims) / factor for i in range(half)], dtype=torch.float64)
    a = pos.to(torch.float64)[:, None, None] * f
    c, s = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def temperature(pos: torch.Tensor, coef: float, every: int) -> torch.Tensor:
    return 1.0 + coef * torch.log(torch.floor((pos.to(torch.float64) + 1.0) / every) + 1.0)


def attend(q: torch.Tensor, K: torch.Tensor, V: torch.Tensor, pos: torch.Tensor, scale: float, window: int = 0,
           sink: Optional[torch.Tensor] = None) -> torch.Tensor:
    """q [T, H, dim] at positions pos over K [n, G, dim], V [n, G, vd] of positions 0 .. n - 1; query head h reads
    key/value head h // (H / G).  window 0: all j <= i; sink [H]: exp(sink) joins the denominator."""
    T, H, G = q.shape[0], q.shape[1], K.shape[1]
    dist = pos[:, None] - torch.arange(K.shape[0])[None, :]
    seen = dist >= 0
    if window > 0:
        seen = seen & (dist < window)
    of_head = torch.arange(H) // (H // G)                                # the key/value head of every query head
    s = (torch.einsum("thd,nhd->htn", q, K[:, of_head]) * scale).masked_fill(~seen, -math.inf)
    if sink is not None:
        s = torch.cat([s, sink[:, None, None].expand(H, T, 1)], dim=2)
    p = torch.exp(s - s.max(dim=2, keepdim=True).values)
    p = p / p.sum(dim=2, keepdim=True)
    return torch.einsum("htn,nhv->thv", p[:, :, : K.shape[0]], V[:, of_head])


def _grow(st: Dict[str, torch.Tensor], key: str, new: torch.Tensor) -> torch.Tensor:
    st[key] = torch.cat([st[key], new]) if key in st else new
    return st[key]


def left_half(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, pos: torch.Tensor, st: Dict) -> torch.Tensor:
    H, G, dim = int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    T = h.shape[0]
    q = (apply(w["q"], h) + w["q.b"]).reshape(T, H, dim)
    k = (apply(w["k"], h) + w["k.b"]).reshape(T, G, dim)
    if m.get("q_temp"):
        q = q * temperature(pos, float(m["q_temp"]["coef"]), int(m["q_temp"]["every"])).to(q.dtype)[:, None, None]
    K = _grow(st, "k", k)
    o = attend(q, K, K, pos, float(m["scale"]), 0, w["sink"])
    o = o * torch.sigmoid(apply(w["g"], h))[:, :, None]
    return apply(w["o"], o.reshape(T, H * dim)) + w["o.b"]


def matrix_memory(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, i: torch.Tensor, f: torch.Tensor, S: torch.Tensor,
                  n: torch.Tensor, m: torch.Tensor) -> torch.Tensor:
    """q (scaled), k [T, heads, dim], v [T, heads, vd], i, f [T, heads]; S [heads, dim, vd], n [heads, dim] and m [heads]
    are carried in place."""
    out = torch.zeros_like(v)
    for t in range(q.shape[0]):
        m_new = torch.maximum(f[t] + m, i[t])
        keep, write = torch.exp(f[t] + m - m_new), torch.exp(i[t] - m_new)
        S.copy_(keep[:, None, None] * S + write[:, None, None] * k[t][:, :, None] * v[t][:, None, :])
        n.copy_(keep[:, None] * n + write[:, None] * k[t])
        m.copy_(m_new)
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out[t] = (S * q[t][:, :, None]).sum(1) / den[:, None]
    return out


def right_half(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float, st: Dict) -> torch.Tensor:
    H, dim, vd, cap = int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["gate_cap"])
    T = h.shape[0]
    q = (apply(w["q"], h)).reshape(T, H, dim) * dim ** -0.5
    k = (apply(w["k"], h)).reshape(T, H, dim)
    v = (apply(w["v"], h)).reshape(T, H, vd)
    i = cap * torch.tanh((h @ w["i"].T + w["i.b"]) / cap)
    f = log_sigmoid(cap * torch.tanh((h @ w["f"].T + w["f.b"]) / cap))
    if "S" not in st:
        st["S"], st["n"], st["m"] = (torch.zeros(H, dim, vd, dtype=h.dtype), torch.zeros(H, dim, dtype=h.dtype),
                                     torch.zeros(H, dtype=h.dtype))
    o = matrix_memory(q, k, v, i, f, st["S"], st["n"], st["m"])
    o = norm(o, w["norm"].reshape(H, vd), eps).reshape(T, H * vd)
    return apply(w["o"], o * torch.sigmoid(apply(w["g"], h)))


def parallel_mixer(h, wl, wr, ml, mr, pos, eps, st) -> torch.Tensor:
    a = left_half(h, wl, ml, pos, st.setdefault("left", {}))
    b = right_half(h, wr, mr, eps, st.setdefault("right", {}))
    return (norm(a, wl["out"], eps) + norm(b, wr["out"], eps)) / 2.0


def gated_scan(u: torch.Tensor, r: torch.Tensor, i: torch.Tensor, lam: torch.Tensor, S: torch.Tensor) -> torch.Tensor:
    """u, r, i [T, width] (r, i after their sigmoids); S [width] is carried in place."""
    out = torch.zeros_like(u)
    for t in range(u.shape[0]):
        log_a = -8.0 * r[t] * softplus(lam)
        S.copy_(torch.exp(log_a) * S + torch.sqrt(-torch.expm1(2.0 * log_a)) * i[t] * u[t])
        out[t] = S
    return out


def block_map(u: torch.Tensor, M: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """u [T, width] in equal parts, each through its own square matrix M[part] [out, in]."""
    nb, n = M.shape[0], M.shape[1]
    return torch.cat([u[:, j * n: (j + 1) * n] @ M[j].T + b[j] for j in range(nb)], dim=1)


def rglru_mixer(h: torch.Tensor, w: Dict[str, torch.Tensor], st: Dict) -> torch.Tensor:
    y = gelu_tanh(apply(w["y"], h) + w["y.b"])
    u = short_filter(apply(w["x"], h) + w["x.b"], w["conv"], st, "taps") + w["conv.b"]
    r = torch.sigmoid(block_map(u, w["ra"], w["ra.b"]))
    i = torch.sigmoid(block_map(u, w["ri"], w["ri.b"]))
    if "S" not in st:
        st["S"] = torch.zeros(u.shape[1], dtype=h.dtype)
    return apply(w["o"], gated_scan(u, r, i, w["lam"], st["S"]) * y)


def attention_mixer(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, pos: torch.Tensor, eps: float,
                    st: Dict) -> torch.Tensor:
    H, G, dim, vd = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    T = h.shape[0]
    q, k, v = (short_filter(apply(w[c], h) + w[c + ".b"], w[c + ".conv"], st, c + ".taps") for c in "qkv")
    q = norm(q.reshape(T, H, dim), w["q.norm"], eps)
    k = norm(k.reshape(T, G, dim), w["k.norm"], eps)
    rot = m.get("rot")
    if rot and int(rot["dims"]):
        factor = float((rot.get("scaling") or {}).get("factor", 1.0))
        q, k = (turn(z, pos, float(rot["base"]), int(rot["dims"]), factor) for z in (q, k))
    K, V = _grow(st, "k", k), _grow(st, "v", v.reshape(T, G, vd))
    o = attend(q, K, V, pos, float(m["scale"]), int((m.get("mask") or {}).get("size") or 0))
    return apply(w["o"], o.reshape(T, H * vd))


def route(z: torch.Tensor, top: int, n_groups: int, keep: int, factor: float):
    """(chosen ids [T, top], weights [T, top]) of router logits z [T, experts]."""
    s = torch.sigmoid(z)
    T, E = s.shape
    c = s.clone()
    if n_groups > 1:
        g = s.reshape(T, n_groups, E // n_groups)
        score = g.topk(min(2, E // n_groups), dim=-1).values.sum(-1)
        alive = torch.zeros(T, n_groups, dtype=torch.bool)
        alive.scatter_(1, score.topk(keep, dim=-1).indices, True)
        c = c.masked_fill(~alive.repeat_interleave(E // n_groups, dim=1), -math.inf)
    ids = c.topk(top, dim=-1).indices
    chosen = s.gather(1, ids)
    return ids, chosen / (chosen.sum(-1, keepdim=True) + 1e-20) * factor


def relu_squared_ff(h: torch.Tensor, up: torch.Tensor, down: torch.Tensor) -> torch.Tensor:
    return apply(down, torch.clamp(apply(up, h), min=0.0) ** 2)


def moe_ff(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict) -> torch.Tensor:
    r = m["router"]
    grp = r.get("groups") or {}
    ids, wts = route(h @ w["router"].T, int(r["top"]), int(grp.get("count") or 1), int(grp.get("keep") or 1),
                     float(r.get("scale", 1.0)))
    out = torch.zeros_like(h)
    for e in range(int(r["experts"])):
        rows, k = (ids == e).nonzero(as_tuple=True)
        if rows.numel():
            out[rows] += wts[rows, k][:, None] * relu_squared_ff(h[rows], w[f"e{e}.up"], w[f"e{e}.down"])
    if m.get("shared"):
        out = out + relu_squared_ff(h, w["shared.up"], w["shared.down"])
    return out


def layer_runs(config: dict) -> List[tuple]:
    """(layer, pass or None, whether a pass starts with it) in running order."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, None, False) for i in range(n)]
    a, b = int(loop["start"]), int(loop["stop"])
    out = [(i, None, False) for i in range(a)]
    for t in range(int(loop["times"])):
        out += [(i, t, i == a) for i in range(a, b)]
    return out + [(i, None, False) for i in range(b, n)]


class Palulorn:
    def __init__(self, config: dict, tensors: Dict[str, torch.Tensor], dtype: torch.dtype = torch.float64):
        self.config, self.dtype = config, dtype
        self.w = {k: v.to(dtype) for k, v in tensors.items()}
        self.eps = float(config["norm"]["eps"])

    def sub(self, prefix: str) -> Dict[str, torch.Tensor]:
        return {k[len(prefix):]: v for k, v in self.w.items() if k.startswith(prefix)}

    def new_state(self) -> dict:
        return {"pos": 0, "runs": [{} for _ in layer_runs(self.config)]}

    def forward(self, tokens: List[int], state: dict, layer_out: Optional[list] = None) -> torch.Tensor:
        """Logits [T, vocab] of the next tokens of a sequence; `state` carries it on."""
        w, cfg, eps = self.w, self.config, self.eps
        pos = torch.arange(state["pos"], state["pos"] + len(tokens))
        x0 = w["embed"][torch.tensor(tokens)] * float((cfg.get("embedding") or {}).get("scale", 1.0))
        x = x0
        for (i, t, starts), st in zip(layer_runs(cfg), state["runs"]):
            L, p = cfg["layers"][i], f"l{i}."
            if starts:
                x = torch.cat([x, x0], dim=-1) @ w["loop.in"].T + w["loop.step"][t]
            h = norm(x, w[p + "norm1"], eps)
            if L["type"] == "parallel":
                y = parallel_mixer(h, self.sub(p + "mix.left."), self.sub(p + "mix.right."), L["mixer"]["left"],
                                   L["mixer"]["right"], pos, eps, st)
            elif L["type"] == "rglru":
                y = rglru_mixer(h, self.sub(p + "mix."), st)
            else:
                y = attention_mixer(h, self.sub(p + "mix."), L["mixer"], pos, eps, st)
            x = x + y
            if L.get("mlp") is not None:
                x = x + moe_ff(norm(x, w[p + "norm2"], eps), self.sub(p + "mlp."), L["mlp"])
            if layer_out is not None:
                layer_out.append(x.clone())
        state["pos"] += len(tokens)
        return norm(x, w["final.norm"], eps) @ w["head"].T
