"""A plain, slow implementation of the Mevulix decoder: whole sequences, float64, one function per mechanism,
written from the design's equations and sharing no code with the package.

``rnd`` is a hook that the caller may set to a rounding function (for instance to bfloat16 and back): it is applied
where a narrower run rounds (the operands of matrix products), so that two runs with and without it estimate that
run's rounding noise.  Everything that the design computes in 32-bit is left alone.
"""
from __future__ import annotations

import math
from typing import Callable, Dict, List, Optional

import torch

F = torch.float64
Round = Optional[Callable[[torch.Tensor], torch.Tensor]]


def _r(x: torch.Tensor, rnd: Round) -> torch.Tensor:
    return x if rnd is None else rnd(x)


def _lin(x: torch.Tensor, w: torch.Tensor, rnd: Round, b: Optional[torch.Tensor] = None) -> torch.Tensor:
    y = _r(x, rnd) @ w.to(F).T
    return y if b is None else y + b.to(F)


# ---- norms and activations -----------------------------------------------------------------------------------
def rms_norm(x, g, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * g.to(F)


def layer_norm(x, g, b, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * g.to(F) + b.to(F)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


# ---- rotation with stretched frequencies -----------------------------------------------------------------------
def frequencies(base: float, dims: int, scaling: Optional[dict]) -> List[float]:
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling is None:
        return f

    def place(turns):
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(place(scaling["fast"])), 0)
    hi = min(math.ceil(place(scaling["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / scaling["factor"] * ramp + fi * (1.0 - ramp))
    return out


def rotate_pairs(x, positions, rot: Optional[dict]):
    """x [T, ..., d]: the neighbours (2i, 2i + 1) of the first ``dims`` elements turn by position * f_i, and grow by the
    factor on cos and sin."""
    if not rot or rot["dims"] == 0:
        return x
    dims, scaling = rot["dims"], rot.get("scaling")
    a = positions.to(F)[:, None] * torch.tensor(frequencies(rot["base"], dims, scaling), dtype=F)
    while a.dim() < x.dim():
        a = a.unsqueeze(1)
    grow = 1.0 if scaling is None else 0.1 * math.log(scaling["factor"]) + 1.0
    cs, sn = grow * torch.cos(a), grow * torch.sin(a)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    turned = torch.stack([u * cs - v * sn, v * cs + u * sn], dim=-1).flatten(-2)
    return torch.cat([turned, x[..., dims:]], dim=-1)


# ---- latent attention ------------------------------------------------------------------------------------------
def queries(h, p, m, eps, rnd: Round = None):
    """q [T, H, dim + rot_dim]: two matrices with a norm between them; the last rot_dim turned."""
    T = h.shape[0]
    c_q = rms_norm(_lin(h, p["dq"], rnd), p["dq.norm"], eps)
    q = _lin(c_q, p["uq"], rnd).view(T, m["heads"], m["dim"] + m["rot_dim"])
    return torch.cat([q[..., :m["dim"]], rotate_pairs(q[..., m["dim"]:], torch.arange(T), m.get("rot"))], dim=-1)


def latent_rows(h, p, m, eps, rnd: Round = None):
    """(c [T, kv_rank], r [T, rot_dim]): what a token leaves behind for all heads."""
    rank = m["kv_rank"]
    dkv = _lin(h, p["dkv"], rnd)
    return rms_norm(dkv[:, :rank], p["dkv.norm"], eps), rotate_pairs(dkv[:, rank:], torch.arange(h.shape[0]), m.get("rot"))


def causal(s):
    """Scores of later keys struck out."""
    T = s.shape[-1]
    return s.masked_fill(~torch.ones(T, T, dtype=torch.bool).tril()[None], -math.inf)


def latent_attention(h, p: Dict[str, torch.Tensor], m: dict, eps: float, rnd: Round = None):
    """h [T, width] of one sequence from position 0; keys and values are rebuilt from the latent row per head."""
    T = h.shape[0]
    H, dim, vd = m["heads"], m["dim"], m["vdim"]
    q = queries(h, p, m, eps, rnd)
    c, r = latent_rows(h, p, m, eps, rnd)
    c, r = _r(c, rnd), _r(r, rnd)
    k = _lin(c, p["uk"], rnd).view(T, H, dim)
    v = _lin(c, p["uv"], rnd).view(T, H, vd)
    s = torch.einsum("thd,shd->hts", _r(q[..., :dim], rnd), _r(k, rnd)) \
        + torch.einsum("thd,sd->hts", _r(q[..., dim:], rnd), r)
    w = torch.softmax(causal(s * m["scale"]), dim=-1)
    return _lin(torch.einsum("hts,shd->thd", w, _r(v, rnd)).reshape(T, H * vd), p["o"], rnd)


# ---- attention with a bias by distance -------------------------------------------------------------------------
def bucket(n: int, rows: int, reach: float) -> int:
    """The row of the bias table for a key ``n`` tokens back: one row each for the nearest ones, then rows that cover
    ever longer stretches up to ``reach``.  The edges are found with whole numbers, so that a distance that lies
    exactly on one falls on its own side of it."""
    half = rows // 2
    if n < half:
        return n
    # half + k rows: (n / half)^(rows - half) >= (reach / half)^k
    k, steps = 0, rows - half
    from fractions import Fraction
    have, unit = (Fraction(n) / half) ** steps, Fraction(reach) / half
    while half + k + 1 <= rows - 1 and have >= unit ** (k + 1):
        k += 1
    return min(rows - 1, half + k)


def temperature(positions, q_temp):
    return torch.tensor([1.0 + q_temp["coef"] * math.log((p + 1) // q_temp["every"] + 1) for p in positions.tolist()], dtype=F)


def attention_queries(h, p, m, eps, rnd: Round = None):
    T = h.shape[0]
    q = rms_norm(_lin(h, p["q"], rnd, p["q.b"]), p["q.norm"], eps) * temperature(torch.arange(T), m["q_temp"])[:, None]
    return q.view(T, m["heads"], m["dim"])


def keys_and_values(h, p, m, eps, rnd: Round = None):
    T, G = h.shape[0], m["kv_heads"]
    k = rms_norm(_lin(h, p["k"], rnd, p["k.b"]), p["k.norm"], eps).view(T, G, m["dim"])
    v = _lin(h, p["v"], rnd, p["v.b"]).view(T, G, m["vdim"])
    return _r(k, rnd), _r(v, rnd)


def weights_with_sink(s, sink):
    """s [H, T, T] causal scores, sink [H]: exp(s_ij) over (exp(sink) + the sum over the row)."""
    sink = sink.to(F)[:, None]
    mx = torch.maximum(s.max(-1).values, sink)
    e = torch.exp(s - mx[..., None])
    return e / (e.sum(-1) + torch.exp(sink - mx))[..., None]


def scores(q, k, p, m):
    """[H, T, T]: scaled, capped, then the bias of the distance."""
    T, H = q.shape[0], m["heads"]
    kk = k.repeat_interleave(H // m["kv_heads"], dim=1)
    s = torch.einsum("thd,shd->hts", q, kk) * m["scale"]
    s = m["softcap"] * torch.tanh(s / m["softcap"])
    rel = p["rel"].to(F)
    by_distance = torch.stack([rel[bucket(n, rel.shape[0], m["bias_max"])] for n in range(T)])      # [T, H]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return s + by_distance[(i - j).clamp(min=0)].permute(2, 0, 1)


def attention(h, p: Dict[str, torch.Tensor], m: dict, eps: float, rnd: Round = None, kv=None):
    """``kv``: (keys, values) of another layer of this kind; without it the layer's own.  Returns (result, keys and
    values read)."""
    T, H, G, vd = h.shape[0], m["heads"], m["kv_heads"], m["vdim"]
    k, v = keys_and_values(h, p, m, eps, rnd) if kv is None else kv
    q = _r(attention_queries(h, p, m, eps, rnd), rnd)
    w = weights_with_sink(causal(scores(q, k, p, m)), p["sink"])
    o = torch.einsum("hts,shd->thd", w, v.repeat_interleave(H // G, dim=1))
    return _lin(o.reshape(T, H * vd), p["o"], rnd), (k, v)


# ---- feed-forwards ---------------------------------------------------------------------------------------------
def dense(h, p, rnd: Round = None):
    return _lin(gelu_tanh(_lin(h, p["gate"], rnd)) * _lin(h, p["up"], rnd), p["down"], rnd)


def expert(h, p, rnd: Round = None, prefix: str = ""):
    return _lin(silu(_lin(h, p[prefix + "gate"], rnd)) * _lin(h, p[prefix + "up"], rnd), p[prefix + "down"], rnd)


def route(z, top, margins: Optional[list] = None):
    """z [T, E]: the ``top`` largest sigmoids are chosen and weigh as they are.  Returns a dense [T, E] matrix.
    ``margins``: a list that gets, per token, how far the last chosen logit lies above the first one left out."""
    s = torch.sigmoid(z)
    if margins is not None and top < z.shape[-1]:
        ranked = torch.sort(z, dim=-1, descending=True).values
        margins.append(ranked[:, top - 1] - ranked[:, top])
    best = torch.topk(z, top, dim=-1).indices
    return torch.zeros_like(z).scatter(1, best, torch.gather(s, 1, best))


def moe(h, p, mlp, rnd: Round = None, margins: Optional[list] = None):
    """An expert works on its INPUT times the router's weight (an expert without input gives nothing)."""
    r = mlp["router"]
    w = route(_lin(h, p["router"], rnd), r["top"], margins)
    y = sum(expert(w[:, e:e + 1] * h, p, rnd, f"e{e}.") for e in range(r["experts"]))
    if mlp.get("shared"):
        y = y + expert(h, p, rnd, "shared.")
    return y


# ---- a layer ---------------------------------------------------------------------------------------------------
def join(x, y, g, b, ls, eps):
    """x plus the sublayer's result, normed and scaled element by element."""
    return x + ls.to(F) * layer_norm(y, g, b, eps)


def sub(tensors: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def layer(x, i: int, tensors, cfg, rnd: Round = None, margins: Optional[list] = None, held: Optional[dict] = None):
    """``held``: keys and values of the attention layers before this one, by layer."""
    L, eps = cfg["layers"][i], cfg["norm"]["eps"]
    t, m = sub(tensors, f"l{i}."), L["mixer"]
    held = {} if held is None else held
    if L["type"] == "attention":
        src = m.get("kv_from")
        y, held[i] = attention(x, sub(t, "mix."), m, eps, rnd, None if src is None else held[src])
    else:
        y = latent_attention(x, sub(t, "mix."), m, eps, rnd)
    x = join(x, y, t["norm1"], t["norm1.b"], t["ls1"], eps)
    mlp = L.get("mlp")
    if mlp is None:
        return x
    p = sub(t, "mlp.")
    y = dense(x, p, rnd) if mlp["kind"] == "dense" else moe(x, p, mlp, rnd, margins)
    return join(x, y, t["norm2"], t["norm2.b"], t["ls2"], eps)


def forward(tokens, tensors, cfg, rnd: Round = None, keep_layers: bool = False, margins: Optional[list] = None):
    """Logits [T, vocab] of one sequence from its first token; with ``keep_layers`` also the stream after every
    layer; ``margins`` collects the routers' margins (see ``route``)."""
    x = tensors["embed"].to(F)[torch.tensor(list(tokens))]
    kept, held = [], {}
    for i in range(len(cfg["layers"])):
        x = layer(x, i, tensors, cfg, rnd, margins, held)
        kept.append(x)
    f = layer_norm(x, tensors["final.norm"], tensors["final.norm.b"], cfg["norm"]["eps"])
    logits = _lin(f, tensors["head"], rnd) * cfg["logit_scale"]
    return (logits, torch.stack(kept)) if keep_layers else logits


def greedy(tokens, tensors, cfg, n_new: int) -> List[int]:
    """``n_new`` tokens, each the largest logit after everything before it (the whole sequence is run again)."""
    seq, out = list(tokens), []
    for _ in range(n_new):
        nxt = int(forward(seq, tensors, cfg)[-1].argmax())
        seq.append(nxt)
        out.append(nxt)
    return out
