"""The plain Mevulix implementation against closed forms (no GPU), and the parts of the package that need no GPU: the
configuration reader, the name table, the cache's plan, the table of distances, what is folded when weights are loaded,
and the command line."""
import json
import math

import pytest
import torch

import mevulix_configs as MC
import plain_mevulix as P
from mevulix_configs import CONFIGS, MEV_A, MEV_B, MEV_C, MEV_D

F64 = torch.float64


def rnd(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed + sum(shape)), dtype=F64)


def test_layer_norm_and_gelu():
    x = torch.tensor([[1.0, 3.0]], dtype=F64)
    y = P.layer_norm(x, torch.tensor([2.0, 5.0]), torch.tensor([0.5, -1.0]), 0.25)
    assert torch.allclose(y, torch.tensor([[-2.0 / math.sqrt(1.25) + 0.5, 5.0 / math.sqrt(1.25) - 1.0]], dtype=F64))
    z = rnd(50)
    assert torch.allclose(P.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"))


def test_rotation_turns_neighbours_and_grows_by_the_scalings_factor():
    x = rnd(3, 2, 10)
    pos = torch.tensor([0, 5, 9])
    y = P.rotate_pairs(x, pos, {"base": 100.0, "dims": 8})
    assert torch.equal(y[..., 8:], x[..., 8:]) and torch.equal(y[0], x[0])
    a = 5 * 100.0 ** (-2 * 1 / 8)
    assert torch.allclose(y[1, :, 2], x[1, :, 2] * math.cos(a) - x[1, :, 3] * math.sin(a))
    assert torch.allclose(y[1, :, 3], x[1, :, 3] * math.cos(a) + x[1, :, 2] * math.sin(a))
    s = {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}
    z = P.rotate_pairs(x, pos, {"base": 100.0, "dims": 8, "scaling": s})
    assert torch.allclose(z[0, :, :8], (0.1 * math.log(4.0) + 1.0) * x[0, :, :8])


def test_stretched_frequencies_keep_the_fast_pairs_and_divide_the_slow_ones():
    s = {"factor": 8.0, "original": 2000, "fast": 32.0, "slow": 1.0}
    f, plain = P.frequencies(1e4, 64, s), P.frequencies(1e4, 64, None)

    def place(t):
        return 64 * math.log(2000 / (2 * math.pi * t)) / (2 * math.log(1e4))
    lo, hi = math.floor(place(32.0)), math.ceil(place(1.0))
    assert 0 < lo < hi < 31
    assert f[:lo + 1] == plain[:lo + 1] and all(math.isclose(a, b / 8.0) for a, b in zip(f[hi:], plain[hi:]))
    mid = (lo + hi) // 2
    ramp = (mid - lo) / (hi - lo)
    assert math.isclose(f[mid], plain[mid] / 8.0 * ramp + plain[mid] * (1 - ramp))
    assert P.frequencies(1e4, 64, dict(s, factor=1.0)) == pytest.approx(plain)


def test_buckets_of_distances():
    assert [P.bucket(n, 8, 64) for n in (0, 1, 2, 3, 4, 7, 8, 15, 16, 31, 32, 63, 64, 10 ** 6)] == [0, 1, 2, 3, 4, 4, 5, 5, 6, 6, 7, 7, 7, 7]
    assert [P.bucket(n, 2, 20) for n in range(5)] == [0, 1, 1, 1, 1]
    assert [P.bucket(n, 9, 33) for n in range(4)] == [0, 1, 2, 3]
    # away from the edges: the formula in floating point
    for rows, reach in ((12, 40), (32, 100), (31, 500), (64, 2000), (3, 7)):
        h = rows // 2
        for n in range(h, 3 * reach):
            b = math.log(n / h) / math.log(reach / h) * (rows - h)
            if abs(b - round(b)) > 1e-9:
                assert P.bucket(n, rows, reach) == min(rows - 1, h + math.floor(b)), (rows, reach, n)


def test_query_temperature_steps():
    t = P.temperature(torch.tensor([0, 2, 3, 4, 7, 100]), {"coef": 0.5, "every": 4})
    want = [1.0, 1.0] + [1.0 + 0.5 * math.log(k) for k in (2, 2, 3, 26)]
    assert torch.allclose(t, torch.tensor(want, dtype=F64))


def _att_weights(m, W, rows=4):
    H, G, dk, dv = (m[k] for k in ("heads", "kv_heads", "dim", "vdim"))
    p = {"q": rnd(H * dk, W), "k": rnd(G * dk, W, seed=1), "v": rnd(G * dv, W, seed=2), "o": torch.eye(H * dv, dtype=F64),
         "q.b": rnd(H * dk, seed=3), "k.b": rnd(G * dk, seed=4), "v.b": rnd(G * dv, seed=5), "rel": rnd(rows, H, seed=6),
         "q.norm": 1 + 0.2 * rnd(H * dk, seed=7), "k.norm": 1 + 0.2 * rnd(G * dk, seed=8), "sink": rnd(H, seed=9)}
    return p


ATT = {"heads": 2, "kv_heads": 1, "dim": 4, "vdim": 3, "scale": 0.6, "softcap": 2.0, "q_temp": {"coef": 0.5, "every": 2}, "bias_max": 5}


def test_attention_by_hand_cap_before_bias_and_a_sink_that_has_neither():
    W, T = 6, 7
    p, h = _att_weights(ATT, W), rnd(T, W, seed=20)
    y, (k, v) = P.attention(h, p, ATT, 1e-12)
    i = 5
    q = h[i] @ p["q"].T + p["q.b"]
    q = q / q.pow(2).mean().sqrt() * p["q.norm"] * (1 + 0.5 * math.log(4))          # floor(6 / 2) + 1
    for head in (0, 1):
        e = []
        for j in range(i + 1):
            kj = h[j] @ p["k"].T + p["k.b"]
            kj = kj / kj.pow(2).mean().sqrt() * p["k.norm"]
            s = (q[4 * head:4 * head + 4] * kj).sum() * 0.6
            row = [0, 1, 2, 2, 3, 3][i - j]                    # 2 ln(n / 2) / ln(5 / 2): 0, 0.88, 1.51 -> rows 2, 2, 3
            e.append(torch.exp(2.0 * torch.tanh(s / 2.0) + p["rel"][row, head]))
        den = sum(e) + torch.exp(p["sink"][head])
        want = sum(w / den * (h[j] @ p["v"].T + p["v.b"]) for j, w in enumerate(e))
        assert torch.allclose(y[i, 3 * head:3 * head + 3], want)
    h2 = h.clone()
    h2[4] += 1.0
    assert ((P.attention(h2, p, ATT, 1e-12)[0] - y).abs().sum(-1) > 1e-9).tolist() == [i >= 4 for i in range(T)]
    # another layer's keys and values: its own do not matter
    other = dict(p, k=rnd(4, W, seed=70), v=rnd(3, W, seed=71))
    assert torch.equal(P.attention(h, other, ATT, 1e-12, kv=(k, v))[0], y)


def test_latent_attention_first_token_and_causality():
    m = {"heads": 2, "dim": 4, "rot_dim": 4, "vdim": 3, "kv_rank": 6, "q_rank": 5, "scale": 0.4, "rot": {"dims": 4, "base": 100.0}}
    W, T = 8, 7
    p = {"dq": rnd(5, W), "dq.norm": 1 + 0.2 * rnd(5, seed=1), "uq": rnd(16, 5), "dkv": rnd(10, W, seed=2),
         "dkv.norm": 1 + 0.2 * rnd(6, seed=3), "uk": rnd(8, 6, seed=4), "uv": rnd(6, 6, seed=5), "o": rnd(W, 6, seed=7)}
    h = rnd(T, W, seed=9)
    y = P.latent_attention(h, p, m, 1e-12)
    c, _ = P.latent_rows(h[:1], p, m, 1e-12)
    assert torch.allclose(y[0], (c @ p["uv"].T @ p["o"].T)[0])             # the first token sees itself alone
    h2 = h.clone()
    h2[4] += 1.0
    assert ((P.latent_attention(h2, p, m, 1e-12) - y).abs().sum(-1) > 1e-9).tolist() == [i >= 4 for i in range(T)]
    assert torch.allclose(P.latent_attention(h, dict(p, dq=7.0 * p["dq"]), m, 1e-12), y)


def test_router_weights_are_the_chosen_sigmoids_and_multiply_the_experts_input():
    z = torch.tensor([[2.0, 0.5, -1.0, 1.0]], dtype=F64)
    s = torch.sigmoid(z[0])
    assert torch.allclose(P.route(z, 2)[0], torch.stack([s[0], s[0] * 0, s[0] * 0, s[3]]))
    W = 4
    mlp = {"router": {"experts": 2, "top": 1}, "shared": {"ff": 2}}
    p = {"router": torch.stack([torch.zeros(W, dtype=F64), torch.ones(W, dtype=F64)])}
    for n, f in (("e0", 3), ("e1", 3), ("shared", 2)):
        p.update({n + ".gate": rnd(f, W, seed=len(n)), n + ".up": rnd(f, W, seed=2), n + ".down": rnd(W, f, seed=3)})
    h = rnd(5, W).abs()
    w = torch.sigmoid(h.sum(-1, keepdim=True))
    want = P.expert(w * h, p, prefix="e1.") + P.expert(h, p, prefix="shared.")
    assert torch.allclose(P.moe(h, p, mlp), want)
    assert not torch.allclose(want, w * P.expert(h, p, prefix="e1.") + P.expert(h, p, prefix="shared."), rtol=0.05)
    assert torch.allclose(P.moe(h, p, {"router": mlp["router"]}), P.expert(w * h, p, prefix="e1."))


def test_config_reader_name_table_and_cache_plan():
    from mivi_v4_b200.cache import KVNeed
    from mivi_v4_b200.config import ConfigError, MevulixConfig
    from mivi_v4_b200.engine.model import Model, describe_config, expected_tensors
    for cfg, _ in CONFIGS.values():
        c = MevulixConfig.from_dict(cfg)
        assert len(c.layers) == len(cfg["layers"]) and c.logit_scale == cfg["logit_scale"] and c.norm_eps == cfg["norm"]["eps"]
    n = {k: tuple(v.shape) for k, v in expected_tensors(MEV_A).items()}
    assert n["embed"] == (97, 96) and n["final.norm"] == (96,) and n["final.norm.b"] == (96,) and n["head"] == (97, 96)
    assert n["l0.norm1"] == n["l0.norm1.b"] == n["l0.norm2.b"] == n["l0.ls1"] == n["l0.ls2"] == (96,)
    assert n["l0.mix.q"] == (192, 96) and n["l0.mix.k.b"] == (64,) and n["l0.mix.v"] == (32, 96) and n["l0.mix.k.norm"] == (64,)
    assert n["l0.mix.rel"] == (12, 6) and n["l0.mix.sink"] == (6,) and n["l0.mix.o"] == (96, 96)
    assert sorted(k for k in n if k.startswith("l2.mix.")) == ["l2.mix." + k for k in ("o", "q", "q.b", "q.norm", "rel", "sink")]
    assert n["l1.mix.dq"] == (24, 96) and n["l1.mix.uq"] == (320, 24) and n["l1.mix.dkv"] == (48, 96) and "l1.mix.sink" not in n
    assert n["l0.mlp.router"] == (6, 96) and n["l0.mlp.e5.down"] == (96, 32) and n["l0.mlp.shared.up"] == (48, 96)
    assert "l0.mlp.shared.sg" not in n and n["l1.mlp.gate"] == (64, 96)
    assert not [k for k in n if k.startswith("l3.") and ("mlp" in k or "norm2" in k or "ls2" in k)]
    assert not [k for k in expected_tensors(MEV_B) if k.startswith("l3.mlp.shared")]
    # how many buckets the bias has is the checkpoint's to say where the configuration does not
    free = json.loads(json.dumps(MEV_A))
    free["layers"][0]["mixer"].pop("bias_rows")
    assert expected_tensors(free)["l0.mix.rel"].shape == (None, 6)
    for cfg, shared in ((MEV_A, {2: 0, 4: 0}), (MEV_C, {3: 1, 4: 2})):
        plan = Model(describe_config(cfg)[1]).cache_plan()
        assert all(isinstance(g.need, KVNeed) for g in plan.groups)
        assert [i for i, o in enumerate(plan.owner) if not o] == sorted(shared)
        assert all(plan.binding[i] == plan.binding[j] for i, j in shared.items())
        # a layer that reads another's keys and values adds no storage
        assert sum(g.n_layers for g in plan.groups) == len(cfg["layers"]) - len(shared)

    def broken(edit, base=MEV_A):
        c = json.loads(json.dumps(base))
        edit(c)
        with pytest.raises(ConfigError):
            MevulixConfig.from_dict(c)
    broken(lambda c: c["layers"][0].update(type="mamba2"))
    broken(lambda c: c["layers"][0]["mixer"].pop("softcap"))
    broken(lambda c: c["layers"][0]["mixer"].update(kv_heads=4))
    broken(lambda c: c["layers"][0]["mixer"]["q_temp"].update(every=0))
    broken(lambda c: c["layers"][0]["mixer"].update(bias_max=0))
    broken(lambda c: c["layers"][0]["mixer"].update(bias_rows=1))
    broken(lambda c: c["layers"][0]["mixer"].update(kv_from=0))          # itself
    broken(lambda c: c["layers"][4]["mixer"].update(kv_from=2))          # a reader
    broken(lambda c: c["layers"][4]["mixer"].update(kv_from=1))          # another kind of layer
    broken(lambda c: c["layers"][4]["mixer"].update(dim=16))
    broken(lambda c: c["layers"][1]["mixer"].pop("q_rank"))
    broken(lambda c: c["layers"][1]["mixer"].pop("rot"))
    broken(lambda c: c["layers"][1]["mixer"]["rot"].update(dims=4))
    broken(lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("slow"))
    broken(lambda c: c["layers"][0]["mlp"]["router"].update(top=7))
    broken(lambda c: c["layers"][0]["mlp"].pop("expert"))
    broken(lambda c: c["layers"][1]["mlp"].update(kind="swiglu"))
    broken(lambda c: c.pop("logit_scale"))
    broken(lambda c: c.update(layers=[]))


def test_the_table_of_distances_is_the_bias_of_every_distance():
    from mivi_v4_b200.parts.mixers import distance_table
    for rows, reach in ((12, 40), (8, 64), (9, 33), (2, 20), (31, 500), (32, 100), (16, 64), (64, 2000), (3, 7), (8, 8), (5, 2.5)):
        rel = rnd(rows, 3, seed=rows).float()
        t = distance_table(rel, reach)
        assert t.shape[0] == 3 and t.shape[1] <= math.ceil(reach) + 1
        for n in range(3 * int(reach) + 5):
            assert torch.equal(t[:, min(n, t.shape[1] - 1)], rel[P.bucket(n, rows, reach)]), (rows, reach, n)
        assert rows == 2 or not torch.equal(t[:, -2], t[:, -1])
    for rows, reach in ((1, 5), (8, 4), (8, 3)):
        with pytest.raises(ValueError):
            distance_table(torch.zeros(rows, 2), reach)


def test_what_is_folded_when_weights_are_loaded():
    from mivi_v4_b200.engine.model import Model, describe_config
    from mivi_v4_b200.weights.random_init import random_tensors
    model = Model(describe_config(MEV_A)[1])
    t = random_tensors(model.named_param_specs(), 3, torch.float32)
    model.load_params(t, torch.float32, "cpu")
    for i, block in enumerate(model.blocks):
        w, b = block.joins[block.mixer_norm]
        assert torch.equal(w, t[f"l{i}.norm1"] * t[f"l{i}.ls1"]) and torch.equal(b, t[f"l{i}.norm1.b"] * t[f"l{i}.ls1"])
        assert (block.ffn is None) == (MEV_A["layers"][i]["mlp"] is None)
    assert torch.allclose(model.final_norm.bias, 0.7 * t["final.norm.b"])
    att = model.blocks[0].mixer
    assert att.b_qkvg.shape[0] == att.w_qkvg.shape[0]
    assert torch.equal(att.b_qkvg[:288], torch.cat([t["l0.mix.q.b"], t["l0.mix.k.b"], t["l0.mix.v.b"]]))
    assert model.blocks[2].mixer.w_qkvg.shape[0] == 192
    # neighbouring pairs of the rotated part become pairs half a part away, in queries and keys alike
    lat, order = model.blocks[1].mixer, [0, 2, 4, 6, 1, 3, 5, 7]
    dkv, uq = t["l1.mix.dkv"], t["l1.mix.uq"].view(10, 32, 24)
    assert torch.equal(lat.w_in[24:72], torch.cat([dkv[:40], dkv[40:][order]]))
    assert torch.equal(lat.w_uq.view(10, 32, 24), torch.cat([uq[:, :24], uq[:, 24:][:, order]], 1))


def test_two_way_routers_stay_far_from_a_close_call(tmp_path):
    """The weights of the bfloat16 engine tests: in every mixture layer the last chosen entry lies well above the
    first one left out."""
    for name, (cfg, seed) in CONFIGS.items():
        c, w = MC.read_folder(MC.write_mevulix(tmp_path, cfg, seed, router="two_way"))
        margins = []
        P.forward(MC.prompts(cfg["vocab"], [150], seed)[0], w, c, margins=margins)
        assert all(float(m.min()) > 0.1 for m in margins), (name, [float(m.min()) for m in margins])


def test_a_changed_constant_a_lost_mechanism_or_another_layers_cache_would_show(tmp_path):
    """The comparison can fail: the plain logits with one mechanism changed lie outside the bfloat16 limit (and so far
    outside the float32 one)."""
    cfg, seed = CONFIGS["A"]
    _, weights = MC.read_folder(MC.write_mevulix(tmp_path, cfg, seed))
    toks = MC.prompts(cfg["vocab"], [60], 5)[0]
    want = P.forward(toks, weights, cfg)
    limit = MC.NOISE_FACTOR * float(MC.noise(cfg, weights, toks, want).median())

    def off(change_cfg=None, change_w=None):
        c, w = json.loads(json.dumps(cfg)), dict(weights)
        if change_cfg:
            change_cfg(c)
        if change_w:
            change_w(w)
        return MC.rel_rms(P.forward(toks, w, c), want)[20:].max().item()

    # (a key lost at the far end, one bucket's edge and the last token of a temperature's step are the kernel tests' matter)
    def mixer(c, i): return c["layers"][i]["mixer"]
    def zero(name): return lambda w: w.update({name: torch.zeros_like(w[name])})
    def one(name): return lambda w: w.update({name: torch.ones_like(w[name])})
    for change in (dict(change_cfg=lambda c: mixer(c, 1)["rot"].update(base=30.0)),
                   dict(change_cfg=lambda c: mixer(c, 1)["rot"].pop("scaling")),
                   dict(change_cfg=lambda c: mixer(c, 1).update(scale=0.2)),
                   dict(change_cfg=lambda c: mixer(c, 0).update(softcap=50.0)),
                   dict(change_cfg=lambda c: mixer(c, 0)["q_temp"].update(coef=0.0)),
                   dict(change_cfg=lambda c: mixer(c, 0)["q_temp"].update(every=25)),
                   dict(change_cfg=lambda c: mixer(c, 0).update(bias_max=30)),
                   dict(change_cfg=lambda c: c["layers"][0]["mlp"].pop("shared")),
                   dict(change_cfg=lambda c: c["layers"][0]["mlp"]["router"].update(top=1)),
                   dict(change_cfg=lambda c: c.update(logit_scale=0.65)),
                   dict(change_w=lambda w: w.update({"l0.mix.sink": torch.full_like(w["l0.mix.sink"], -30.0)})),
                   dict(change_w=lambda w: w.update({"l0.mix.rel": torch.roll(w["l0.mix.rel"], 1, 0)})),
                   dict(change_w=zero("l0.mix.q.b")), dict(change_w=zero("l0.mix.k.b")), dict(change_w=zero("l0.mix.v.b")),
                   dict(change_w=zero("l2.mix.q.b")), dict(change_w=zero("l0.norm1.b")), dict(change_w=zero("l4.norm2.b")),
                   dict(change_w=one("l0.norm2")), dict(change_w=one("l1.ls1")), dict(change_w=one("l1.ls2")),
                   dict(change_w=one("final.norm")), dict(change_w=zero("final.norm.b")), dict(change_w=one("l0.mix.q.norm")),
                   dict(change_w=one("l0.mix.k.norm")), dict(change_w=one("l1.mix.dkv.norm")), dict(change_w=one("l1.mix.dq.norm")),
                   dict(change_w=lambda w: w.update({"l0.mix.k": torch.roll(w["l0.mix.k"], 32, 0)}))):
        assert off(**change) > 1.2 * limit, (off(**change), limit)


def test_command_line_writes_and_describes_a_model_folder(tmp_path, capsys):
    from mivi_v4_b200.cli import main
    cfg = tmp_path / "config.json"
    cfg.write_text(json.dumps(MEV_D))
    out = tmp_path / "model"
    assert main(["random", "--config", str(cfg), "--seed", "1", "--out", str(out)]) == 0
    assert (out / "config.json").is_file() and (out / "model.safetensors").is_file()
    capsys.readouterr()
    assert main(["info", "-m", str(out)]) == 0
    text = capsys.readouterr().out
    assert "architecture: Mevulix" in text and "l1.mix.rel" in text and "l0.mlp.router" in text and "l2.ls1" in text
