"""A plain, slow implementation of the Redisun decoder: whole sequences, float64, one function per mechanism,
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


def _lin(x: torch.Tensor, w: torch.Tensor, rnd: Round) -> torch.Tensor:
    return _r(x, rnd) @ w.to(F).T


# ---- norms ---------------------------------------------------------------------------------------------------
def rms_norm(x, g, eps):
    """x over its root mean square, times ``g``: a weight per coordinate, or ONE number for all of them."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * g.to(F)


# ---- embedding -----------------------------------------------------------------------------------------------
def bigram_rows(tokens: List[int], buckets: int, mul_prev: int, mul_cur: int) -> List[int]:
    """The row of the bigram table for every token of a sequence."""
    return [buckets if i == 0 else (tokens[i - 1] * mul_prev + t * mul_cur) % buckets for i, t in enumerate(tokens)]


def embedding(tokens, embed, bigram, cfg):
    bg = cfg["embedding"]["bigram"]
    rows = bigram_rows(list(tokens), bg["buckets"], bg["mul_prev"], bg["mul_cur"])
    return embed.to(F)[torch.tensor(list(tokens))] + bigram.to(F)[torch.tensor(rows)]


# ---- rotation ------------------------------------------------------------------------------------------------
def rotate_half(x, positions, base, dims):
    """x [T, ..., d]: element i < dims/2 turns with element i + dims/2 by positions * base^(-2i/dims)."""
    if dims == 0:
        return x
    half = dims // 2
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=F)
    a = positions.to(F)[:, None] * f[None, :]
    while a.dim() < x.dim():
        a = a.unsqueeze(1)
    cs, sn = torch.cos(a), torch.sin(a)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * cs - v * sn, v * cs + u * sn, x[..., dims:]], dim=-1)


# ---- latent attention ----------------------------------------------------------------------------------------
def queries(h, p, m, eps, rnd: Round = None):
    """q [T, H, dim + rot_dim]: a low-rank step with a norm between its two matrices; the last rot_dim turned."""
    T = h.shape[0]
    c_q = rms_norm(_lin(h, p["dq"], rnd), p["dq.norm"], eps)
    q = _lin(c_q, p["uq"], rnd).view(T, m["heads"], m["dim"] + m["rot_dim"])
    return torch.cat([q[..., :m["dim"]], rotate_half(q[..., m["dim"]:], torch.arange(T), *_rot(m))], dim=-1)


def _rot(m):
    rot = m.get("rot") or {"base": 1.0, "dims": 0}
    return rot["base"], rot["dims"]


def latent_rows(h, p, m, eps, rnd: Round = None):
    """(c [T, kv_rank], r [T, rot_dim]): what a token leaves behind for all heads."""
    rank = m["kv_rank"]
    dkv = _lin(h, p["dkv"], rnd)
    return rms_norm(dkv[:, :rank], p["dkv.norm"], eps), rotate_half(dkv[:, rank:], torch.arange(h.shape[0]), *_rot(m))


def weights_with_sink(s, sink):
    """s [H, T, T] scores, sink [H]: exp(s_ij) over (exp(sink) + the sum over the row), causal."""
    T = s.shape[-1]
    s = s.masked_fill(~torch.ones(T, T, dtype=torch.bool).tril()[None], -math.inf)
    sink = sink.to(F)[:, None]
    mx = torch.maximum(s.max(-1).values, sink)
    e = torch.exp(s - mx[..., None])
    return e / (e.sum(-1) + torch.exp(sink - mx))[..., None]


def latent_attention(h, p: Dict[str, torch.Tensor], m: dict, eps: float, rnd: Round = None):
    """h [T, width] of one sequence from position 0.  Keys and values are rebuilt from the latent row per head
    (nothing is folded into the queries): the slow form."""
    T = h.shape[0]
    H, dim, vd = m["heads"], m["dim"], m["vdim"]
    q = queries(h, p, m, eps, rnd)
    c, r = latent_rows(h, p, m, eps, rnd)
    k = _lin(c, p["uk"], rnd).view(T, H, dim)
    v = _lin(c, p["uv"], rnd).view(T, H, vd)
    s = torch.einsum("thd,shd->hts", _r(q[..., :dim], rnd), _r(k, rnd)) \
        + torch.einsum("thd,sd->hts", _r(q[..., dim:], rnd), _r(r, rnd))
    w = weights_with_sink(s * m["scale"], p["sink"])
    o = torch.einsum("hts,shd->thd", w, _r(v, rnd))
    o = o * torch.sigmoid(_lin(h, p["g"], rnd))[:, :, None]                # one gate a head
    return _lin(o.reshape(T, H * vd), p["o"], rnd)


# ---- feed-forwards ---------------------------------------------------------------------------------------------
def dense(h, p, rnd: Round = None):
    a = _lin(h, p["gate"], rnd)
    return _lin(a * torch.sigmoid(a) * _lin(h, p["up"], rnd), p["down"], rnd)


def expert(h, p, limit, rnd: Round = None, prefix: str = ""):
    g = torch.clamp(_lin(h, p[prefix + "gate"], rnd), max=limit)
    u = torch.clamp(_lin(h, p[prefix + "up"], rnd), min=-limit, max=limit)
    return _lin(g * torch.sigmoid(1.702 * g) * (u + 1.0), p[prefix + "down"], rnd)


def route(z, top, margins: Optional[list] = None):
    """z [T, E]: the ``top`` largest are chosen, their weights are the softmax over the chosen alone.  Returns a dense
    [T, E] matrix.  ``margins``: a list that gets, per token, how far the last chosen logit lies above the first one
    left out."""
    best = torch.topk(z, top, dim=-1)
    if margins is not None and top < z.shape[-1]:
        ranked = torch.sort(z, dim=-1, descending=True).values
        margins.append(ranked[:, top - 1] - ranked[:, top])
    return torch.zeros_like(z).scatter(1, best.indices, torch.softmax(best.values, dim=-1))


def moe(h, p, mlp, rnd: Round = None, margins: Optional[list] = None):
    r = mlp["router"]
    w = route(_lin(h, p["router"], rnd) + p["router.b"].to(F), r["top"], margins)
    y = sum(w[:, e:e + 1] * expert(h, p, mlp["expert"]["limit"], rnd, f"e{e}.") for e in range(r["experts"]))
    if mlp.get("shared"):
        y = y + expert(h, p, mlp["shared"]["limit"], rnd, "shared.")
    return y


# ---- a layer ---------------------------------------------------------------------------------------------------
def join(x, y, wg, bg, g, alpha, eps, rnd: Round = None):
    """The norm after the sum: norm(alpha x + sigmoid(W x + b) * y), y being the sublayer's result from x."""
    return rms_norm(alpha * x + torch.sigmoid(_lin(x, wg, rnd) + bg.to(F)) * y, g, eps)


def sub(tensors: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def layer(x, i: int, tensors, cfg, rnd: Round = None, margins: Optional[list] = None):
    L, eps, alpha = cfg["layers"][i], cfg["norm"]["eps"], cfg["postln_alpha"]
    t = sub(tensors, f"l{i}.")
    y = latent_attention(x, sub(t, "mix."), L["mixer"], eps, rnd)
    x = join(x, y, t["rg1"], t["rg1.b"], t["norm1"], alpha, eps, rnd)
    mlp = L.get("mlp")
    if mlp is None:
        return x
    p = sub(t, "mlp.")
    y = dense(x, p, rnd) if mlp["kind"] == "dense" else moe(x, p, mlp, rnd, margins)
    return join(x, y, t["rg2"], t["rg2.b"], t["norm2"], alpha, eps, rnd)


def forward(tokens, tensors, cfg, rnd: Round = None, keep_layers: bool = False, margins: Optional[list] = None):
    """Logits [T, vocab] of one sequence from its first token; with ``keep_layers`` also the stream after every
    layer; ``margins`` collects the routers' margins (see ``route``)."""
    x = embedding(tokens, tensors["embed"], tensors["bigram"], cfg)
    kept = []
    for i in range(len(cfg["layers"])):
        x = layer(x, i, tensors, cfg, rnd, margins)
        kept.append(x)
    logits = _lin(rms_norm(x, tensors["final.norm"], cfg["norm"]["eps"]), tensors["head"], rnd)
    return (logits, torch.stack(kept)) if keep_layers else logits


def greedy(tokens, tensors, cfg, n_new: int) -> List[int]:
    """``n_new`` tokens, each the largest logit after everything before it (the whole sequence is run again)."""
    seq, out = list(tokens), []
    for _ in range(n_new):
        nxt = int(forward(seq, tensors, cfg)[-1].argmax())
        seq.append(nxt)
        out.append(nxt)
    return out
