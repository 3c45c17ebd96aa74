"""Small Redisun configurations for the tests, the weights they run with, and the rounding-noise estimate.

The configurations differ from one another in every size, in the order of the layers and in which options are on: one
head and ten heads (more than a block of the attention kernel takes), sizes that are no multiples of 8, latents narrower
and wider than a head, queries' latents of the stream's own width, values of one number, no rotated part, sizes that are
all equal; dense feed-forwards, mixtures with one expert, with all experts chosen, with one chosen, with and without a
shared expert whose width and limit differ from the others', layers without a feed-forward; alphas under and over 1.
Weights are drawn by the library's random-weights writer with its "loud" distributions and then sharpened where a fault
would otherwise hide: sinks, gate and router biases of size one, norm numbers well away from one, limits that cut off a
good part of the pre-activations."""
import os

import torch
from safetensors.torch import load_file, save_file

from votavik_configs import assert_rows, prompts, read_folder, rel_rms, NOISE_FACTOR  # noqa: F401  (generic helpers)


def _att(heads, dim, rot_dim, vdim, rank, q_rank, base, scale, mlp=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank, "scale": scale}
    if rot_dim:
        m["rot"] = {"dims": rot_dim, "base": base}
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, top, ff, limit, shared=None):
    d = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if shared:
        d["shared"] = {"ff": shared[0], "limit": shared[1]}
    return d


def _model(vocab, width, eps, alpha, bigram, layers):
    return {"architecture": "Redisun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "postln_alpha": alpha,
            "embedding": {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))}, "layers": layers}


# A: ten heads, a mixture first, a shared expert with another limit; then a dense layer; then one without feed-forward
RED_A = _model(97, 96, 1e-5, 2.0, (53, 5, 3),
               [_att(10, 24, 8, 16, 40, 24, 100.0, 0.5, _moe(6, 2, 32, 0.9, (48, 1.4))),
                _att(4, 16, 16, 32, 72, 56, 5000.0, 0.6, _dense(64)),
                _att(3, 8, 8, 16, 16, 96, 10.0, 0.4, None)])

# B: nothing is a multiple of 8, one head, one chosen expert, a mixture without a shared expert whose experts are all chosen
RED_B = _model(131, 52, 1e-3, 0.7, (17, 1, 1),
               [_att(1, 10, 6, 7, 20, 13, 1e4, 0.4, _dense(30)),
                _att(3, 5, 2, 12, 9, 7, 100.0, 0.5, _moe(5, 1, 20, 0.6, (12, 0.8))),
                _att(2, 12, 4, 9, 15, 22, 1e3, 0.3, _moe(3, 3, 10, 1.1))])

# C: wide heads, a latent of more than 128 numbers, nine heads, several chosen experts
RED_C = _model(200, 128, 1e-6, 3.5, (1009, 131, 17),
               [_att(2, 64, 32, 64, 136, 48, 5e4, 0.12, _moe(9, 4, 48, 1.0, (16, 0.7))),
                _att(9, 32, 16, 48, 64, 128, 500.0, 0.2, _dense(80)),
                _att(8, 40, 24, 32, 32, 40, 1e6, 0.15, _moe(4, 3, 16, 2.0, (64, 2.0)))])

# D: sizes that are all equal, values of one number, no rotated part, one expert, one bucket, alpha 1
RED_D = _model(40, 40, 1e-5, 1.0, (1, 2, 9),
               [_att(1, 8, 8, 8, 40, 40, 100.0, 0.5, _moe(1, 1, 40, 0.8, (40, 0.8))),
                _att(8, 1, 2, 1, 6, 8, 50.0, 1.0, _dense(40)),
                _att(5, 16, 0, 16, 24, 16, 0.0, 0.3, _dense(16))])

CONFIGS = {"A": (RED_A, 41), "B": (RED_B, 42), "C": (RED_C, 43), "D": (RED_D, 44)}

ROUTE_PUSH = 6.0


def route_direction(cfg, seed):
    """The unit vector of the stream that "two_way" routers read."""
    u = torch.randn(cfg["width"], generator=torch.Generator().manual_seed(1000 + seed))
    return u / u.norm()


def token_sign(vocab):
    """+1 or -1 for every token id, changing every three ids."""
    return 1.0 - 2.0 * ((torch.arange(vocab) // 3) % 2)


def sharpen(weights, cfg, seed, router="random"):
    """Values of size one where the random-weights writer draws small ones.  ``router`` = "random" leaves the routers'
    rows as drawn.  "two_way": every router's rows are multiples of ONE direction u of the stream, with unevenly spaced
    factors, and the token embedding carries ``ROUTE_PUSH`` u with a sign that depends on the token id: u . x stays far
    from zero in every layer, so the order of the logits depends on its sign only, and a bfloat16 run chooses the
    experts that the plain implementation chooses, while tokens still take one of two routes."""
    gen = torch.Generator().manual_seed(seed)
    out = dict(weights)
    u = route_direction(cfg, seed)

    def rand(shape):
        return torch.randn(shape, generator=gen)
    if router == "two_way":
        emb = weights["embed"].float()
        out["embed"] = (emb + ROUTE_PUSH * token_sign(emb.shape[0])[:, None] * u[None, :]).to(weights["embed"].dtype)
    for name, w in weights.items():
        if name.endswith(".sink"):                               # sinks that take a share of the softmax
            out[name] = (2.0 + 1.5 * rand(w.shape)).to(w.dtype)
        elif name.endswith((".rg1.b", ".rg2.b")):
            out[name] = rand(w.shape).to(w.dtype)
        elif name.endswith((".dq.norm", ".dkv.norm")):
            out[name] = (1.0 + 0.4 * rand(w.shape)).to(w.dtype)
        elif name.endswith((".norm1", ".norm2")) or name == "final.norm":
            out[name] = (0.5 + 1.3 * torch.rand(w.shape, generator=gen)).to(w.dtype)
        elif name.endswith(".router.b"):
            out[name] = ((0.8 if router == "random" else 0.05) * rand(w.shape)).to(w.dtype)
        elif name.endswith(".router") and router == "two_way":
            E = w.shape[0]
            factors = (4.0 * torch.linspace(0.0, 1.0, E) ** 1.5 - 1.5)[torch.randperm(E, generator=gen)]
            out[name] = (factors[:, None] * (1.8 * cfg["width"] ** -0.5) * u[None, :]).to(w.dtype)
    return out


def write_redisun(tmpdir, cfg, seed, store="bfloat16", change=None, tag="", router="random"):
    """A model folder for ``cfg``: loud random weights, sharpened; ``change(weights) -> weights`` edits them."""
    from mivi_v4_b200 import write_random_model
    d = os.path.join(str(tmpdir), f"redisun_s{seed}_{store}_{router}{tag}")
    if os.path.isdir(d):
        return d
    write_random_model(d, cfg, seed, store, "loud")
    path = os.path.join(d, "model.safetensors")
    weights = sharpen(load_file(path), cfg, seed, router)
    if change is not None:
        weights = change(weights)
    save_file({k: v.contiguous() for k, v in weights.items()}, path)
    return d


def router_for(dtype):
    return "random" if dtype in (torch.float32, "float32") else "two_way"


def round_to(dtype):
    return lambda x: x.to(dtype).to(torch.float64)


def noise(cfg, weights, tokens, want, dtype=torch.bfloat16):
    """What rounding alone does to each row of the logits in a run of ``dtype``, on ``rel_rms``'s scale, and never
    less than twice the median of that over the rows.  Two samples of every row's sensitivity are taken, the plain
    implementation with the operands of its products rounded to float32 and to bfloat16 (whose unit is 2^15 times
    larger), and the larger one counts."""
    import plain_redisun as P
    in32 = rel_rms(P.forward(list(tokens), weights, cfg, rnd=round_to(torch.float32)), want)
    in16 = rel_rms(P.forward(list(tokens), weights, cfg, rnd=round_to(torch.bfloat16)), want)
    if dtype == torch.float32:
        own, other = in32, in16 * 2.0 ** -15
    else:
        own, other = in16, (in32 * 2.0 ** 15).clamp(max=1.0)
    return torch.maximum(torch.maximum(own, other), 2.0 * own.median())
