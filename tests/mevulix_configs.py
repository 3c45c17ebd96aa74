"""Small Mevulix configurations for the tests, the weights they run with, and the rounding-noise estimate.

The configurations differ from one another in every size, in the order of the layers and in which options are on: one
head and ten heads, sizes that are no multiples of 8, values wider and narrower than keys, bias tables of an odd number
of rows, of two rows, with edges that fall exactly on a distance and with a reach beyond every prompt, layers that read
another layer's keys and values (one directly after it, several from the same one, with a temperature and a bias of their
own), rotations with and without stretched frequencies and none at all, sizes that are all equal; dense feed-forwards,
mixtures with one expert, with all experts chosen, with one chosen, with and without a shared expert, layers without a
feed-forward; factors on the logits under and over 1.  Weights are drawn by the library's random-weights writer with its
"loud" distributions and then sharpened where a fault would otherwise hide: sinks, distance biases and projection biases
of size one, norm weights and the layers' vectors well away from one."""
import os

import torch
from safetensors.torch import load_file, save_file

from votavik_configs import assert_rows, prompts, read_folder, rel_rms, NOISE_FACTOR  # noqa: F401  (generic helpers)


def _lat(heads, dim, rot_dim, vdim, rank, q_rank, base, scale, scaling=None, mlp=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank, "scale": scale}
    if rot_dim:
        m["rot"] = {"dims": rot_dim, "base": base}
        if scaling:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def _att(heads, kv_heads, dim, vdim, scale, softcap, temp, rows, reach, kv_from=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": softcap,
         "q_temp": {"coef": temp[0], "every": temp[1]}, "bias_rows": rows, "bias_max": reach}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, top, ff, shared=None):
    d = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        d["shared"] = {"ff": shared}
    return d


def _model(vocab, width, eps, logit_scale, layers):
    return {"architecture": "Mevulix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale,
            "layers": layers}


# A: an attention layer first, read by the next layer but one and by the last; ten heads in latent attention
MEV_A = _model(97, 96, 1e-5, 0.7,
               [_att(6, 2, 32, 16, 0.3, 5.0, (0.8, 7), 12, 40, mlp=_moe(6, 2, 32, 48)),
                _lat(10, 24, 8, 16, 40, 24, 100.0, 0.6, (4.0, 64, 8.0, 1.0), _dense(64)),
                _att(6, 2, 32, 16, 0.6, 3.0, (0.3, 50), 8, 64, 0, _dense(32)),
                _lat(3, 16, 16, 32, 72, 56, 5000.0, 0.2, (16.0, 4096, 32.0, 1.0), None),
                _att(6, 2, 32, 16, 0.4, 8.0, (1.5, 100), 9, 33, 0, _moe(4, 4, 16))])

# B: nothing is a multiple of 8, one head, one chosen expert, a table of two rows, a rotation that is not stretched
MEV_B = _model(131, 52, 1e-3, 1.9,
               [_lat(1, 10, 6, 7, 20, 13, 1e4, 0.3, None, _dense(30)),
                _att(3, 1, 11, 9, 0.35, 4.0, (1.0, 3), 2, 20, mlp=_moe(5, 1, 20, 12)),
                _att(3, 1, 11, 9, 0.3, 2.5, (0.5, 1), 31, 500, 1, None),
                _lat(3, 5, 2, 12, 9, 7, 100.0, 0.4, (2.0, 30, 3.0, 0.5), _moe(3, 3, 10))])

# C: wide heads, several chosen experts, two attention layers with caches of their own and one reader each
MEV_C = _model(200, 128, 1e-6, 3.0,
               [_lat(2, 64, 32, 64, 136, 48, 5e4, 0.1, (8.0, 512, 32.0, 1.0), _moe(9, 4, 48, 16)),
                _att(8, 4, 64, 64, 0.125, 20.0, (0.4, 64), 32, 100, mlp=_dense(80)),
                _att(4, 4, 16, 128, 0.3, 6.0, (0.6, 20), 16, 64, mlp=_moe(4, 3, 16, 64)),
                _att(8, 4, 64, 64, 0.1, 10.0, (0.2, 200), 20, 300, 1, _moe(3, 1, 64)),
                _att(4, 4, 16, 128, 0.25, 9.0, (0.9, 33), 64, 2000, 2, _dense(128)),
                _lat(9, 32, 16, 48, 64, 128, 500.0, 0.15, (3.0, 100, 4.0, 1.0), _dense(48))])

# D: sizes that are all equal, values of one number, no rotated part, one expert, steps of the temperature at every token
MEV_D = _model(40, 40, 1e-5, 1.0,
               [_lat(1, 8, 8, 8, 40, 40, 100.0, 0.4, (1.0, 100, 2.0, 1.0), _moe(1, 1, 40, 40)),
                _att(8, 8, 8, 8, 0.5, 7.0, (0.5, 1), 8, 8, mlp=_dense(40)),
                _att(8, 8, 8, 8, 0.5, 7.0, (0.5, 1), 8, 8, 1, _moe(2, 1, 40)),
                _lat(8, 1, 0, 1, 6, 8, 0.0, 1.0, None, None)])

CONFIGS = {"A": (MEV_A, 51), "B": (MEV_B, 52), "C": (MEV_C, 53), "D": (MEV_D, 54)}

ROUTE_PUSH = 10.0


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
        elif name.endswith(".rel"):                              # neighbouring buckets that differ
            out[name] = (1.5 * rand(w.shape)).to(w.dtype)
        elif name.endswith((".q.b", ".k.b", ".v.b")):
            out[name] = (0.7 * rand(w.shape)).to(w.dtype)
        elif name.endswith((".norm1.b", ".norm2.b", "final.norm.b")):
            out[name] = (0.3 * rand(w.shape)).to(w.dtype)
        elif name.endswith((".dq.norm", ".dkv.norm", ".q.norm", ".k.norm", ".norm1", ".norm2", "final.norm")):
            out[name] = (1.0 + 0.4 * rand(w.shape)).to(w.dtype)
        elif name.endswith((".ls1", ".ls2")):
            out[name] = (0.5 + 0.5 * torch.rand(w.shape, generator=gen)).to(w.dtype)
        elif name.endswith(".router") and router == "two_way":
            E = w.shape[0]
            factors = (4.0 * torch.linspace(0.0, 1.0, E) ** 1.5 - 1.5)[torch.randperm(E, generator=gen)]
            out[name] = (factors[:, None] * (1.2 * cfg["width"] ** -0.5) * u[None, :]).to(w.dtype)
    return out


def write_mevulix(tmpdir, cfg, seed, store="bfloat16", change=None, tag="", router="random"):
    """A model folder for ``cfg``: loud random weights, sharpened; ``change(weights) -> weights`` edits them."""
    from mivi_v4_b200 import write_random_model
    d = os.path.join(str(tmpdir), f"mevulix_s{seed}_{store}_{router}{tag}")
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
    import plain_mevulix as P
    in32 = rel_rms(P.forward(list(tokens), weights, cfg, rnd=round_to(torch.float32)), want)
    in16 = rel_rms(P.forward(list(tokens), weights, cfg, rnd=round_to(torch.bfloat16)), want)
    if dtype == torch.float32:
        own, other = in32, in16 * 2.0 ** -15
    else:
        own, other = in16, (in32 * 2.0 ** 15).clamp(max=1.0)
    return torch.maximum(torch.maximum(own, other), 2.0 * own.median())
