"""Every kernel that the Redisun decoder added or widened, alone, against the plain implementation's function of the
same mechanism (float64), at sizes of the tests' own: the norm after the residual sum with its gate, the norm of one
number, the per-head products of few and of many tokens with both kinds of gate and the rotation of the queries' tails,
latent attention whose queries come through a latent (any cut, pages in no order, a loud key at page borders and far
away, sinks, both step kinds), the router with a bias and softmax over the chosen logits, the clamped activation on its
own, behind the router's weights and inside every matrix product, the mixture in short, long and sorted steps, the
bigram embedding's rounded rows."""
import functools

import pytest
import torch

import plain_redisun as P

pytestmark = pytest.mark.gpu
F64 = torch.float64
BF = torch.bfloat16
DEV = "cuda:0"
DTYPES = [torch.float32, torch.bfloat16]


def K():
    from mivi_v4_b200.ops import kernels
    return kernels


def rnd(*shape, seed=0, scale=1.0):
    return scale * torch.randn(*shape, generator=torch.Generator().manual_seed(seed + 7 * len(shape) + sum(shape)), dtype=F64)


def dev(x, dtype=torch.float32):
    return x.to(dtype).to(DEV).contiguous()


def i32(xs):
    return torch.tensor(xs, dtype=torch.int32, device=DEV)


def close(got, want, tol=2e-5, what=""):
    got, want = got.detach().double().cpu(), want.double()
    assert got.shape == want.shape, (what, got.shape, want.shape)
    assert torch.isfinite(got).all(), what
    err = (got - want).abs().max().item() / max(want.abs().max().item(), 1e-30)
    assert err <= tol, f"{what}: off by {err:.3g} of the largest value (limit {tol})"


def make_step(lens, starts, dtype, page_rows):
    from mivi_v4_b200.engine.step import StepContext, Workspace
    return StepContext(slots=list(range(len(lens))), starts=starts, token_lists=[[0] * n for n in lens], out_rows=[],
                       page_rows={0: page_rows}, dtype=dtype, ws=Workspace(DEV))


# ------------------------------------------------------------------------------------------ norms
@pytest.mark.parametrize("H,N", [(24, 3), (50, 5), (516, 9), (2048, 2), (4096, 3), (5000, 2), (8, 1)])
def test_norm_after_the_sum_with_and_without_its_gate(H, N):
    k = K()
    x, y, y2, z, b, w = rnd(N, H), rnd(N, H, seed=1), rnd(N, H, seed=2), rnd(N, H, seed=3, scale=2.0), rnd(H, seed=4), 1 + rnd(H, seed=5)
    wide = torch.full((N, H + 12), float("nan"), dtype=F64)
    wide[:, 8:8 + H] = z
    for gate in (None, "own", "slice", "odd slice"):
        for dtype in (None, torch.float32, BF):
            for two in (False, True):
                v = 1.5 * y + (-0.5 * y2 if two else 0.0)
                s = 2.5 * x + (v if gate is None else torch.sigmoid(z + (b if gate != "own" else 0.0)) * v)
                want = s / torch.sqrt((s * s).mean(-1, keepdim=True) + 1e-3) * w
                resid = dev(x)
                rounded = None if dtype is None else torch.full((N, H), float("nan"), dtype=dtype, device=DEV)
                at = 8 if gate == "slice" else 3
                wd = dev(wide)
                if gate == "odd slice":
                    wd[:, 3:3 + H] = dev(z)
                zd = None if gate is None else (dev(z) if gate == "own" else wd[:, at:at + H])
                k.sum_norm(dev(y), resid, 2.5, dev(w), 1e-3, s1=1.5, y2=dev(y2) if two else None, s2=-0.5, gate=zd,
                           gate_bias=dev(b) if gate in ("slice", "odd slice") else None, rounded=rounded)
                close(resid, want, 3e-6, f"gate {gate}, two branches {two}")
                if rounded is not None:
                    assert torch.equal(rounded, resid.to(dtype))


def test_norm_part_of_one_number():
    from mivi_v4_b200.parts import PartSpec, build
    n = build("norm", PartSpec("rmsnorm", dict(dim=200, eps=1e-2, scalar=True)))
    assert n.param_specs()["weight"].shape == ()
    n.load({"weight": torch.tensor(0.37, device=DEV)})
    x = rnd(5, 200)
    out = torch.empty(5, 200, device=DEV)
    n.forward(dev(x), out)
    close(out, P.rms_norm(x, torch.tensor(0.37), 1e-2), 2e-6)


# ------------------------------------------------------------------------------------------ a small matrix per head
@pytest.mark.parametrize("w_dtype", DTYPES)
@pytest.mark.parametrize("N", [1, 7, 8, 9, 64, 65, 130])
@pytest.mark.parametrize("nh,I,O", [(3, 64, 256), (2, 24, 40), (5, 9, 13), (1, 200, 66), (4, 1, 6), (2, 520, 72), (3, 16, 7)])
def test_per_head_products_of_few_and_many_tokens(nh, I, O, N, w_dtype):
    """y[n, h] = W_h x[n, h] and W_h^T x[n, h], plain, with a gate an element and a gate a head, inputs and outputs that
    are slices of wider rows."""
    k = K()
    x = rnd(N, nh, I + 5)
    ge, gh = rnd(N, nh * O, seed=1), rnd(N, nh, seed=2)
    for transposed in (False, True):
        w = rnd(nh * I if transposed else nh * O, O if transposed else I, seed=3, scale=I ** -0.5)
        wr = w.to(w_dtype).double()
        plain = torch.einsum("nhi,hio->nho", x[..., :I], wr.view(nh, I, O)) if transposed else \
            torch.einsum("nhi,hoi->nho", x[..., :I], wr.view(nh, O, I))
        for gate, factor in ((None, 1.0), (ge, torch.sigmoid(ge).view(N, nh, O)), (gh, torch.sigmoid(gh)[:, :, None])):
            for y_dtype, tol in ((torch.float32, 1e-5), (BF, 5e-3)):
                y = torch.full((N, nh, O + 3), float("nan"), dtype=y_dtype, device=DEV)
                k.head_product(dev(x), dev(w, w_dtype), y, nh, I, O, transposed=transposed,
                               gate=None if gate is None else dev(gate))
                close(y[..., :O], plain * factor, tol, f"transposed {transposed}")
                assert torch.isnan(y[..., O:].float()).all()


@pytest.mark.parametrize("N", [3, 8, 70])
@pytest.mark.parametrize("nh,I,O,rot,rot_dims", [(3, 16, 24, 8, 8), (2, 5, 70, 6, 4), (9, 32, 64, 2, 0), (1, 64, 130, 34, 34)])
def test_per_head_products_turn_the_tail(nh, I, O, rot, rot_dims, N):
    from mivi_v4_b200.parts.position import Rope
    k = K()
    x, w = rnd(N, nh, I + rot), rnd(nh * I, O, seed=1)
    pos = torch.tensor([(37 * n) % 1000 for n in range(N)])
    inv = Rope(rot_dims, 1e4, "half_split").rotary(DEV)[0] if rot_dims else None
    y = torch.full((N, nh, O + rot), float("nan"), device=DEV)
    k.head_product(dev(x), dev(w), y, nh, I, O, transposed=True, rot=rot, rot_dims=rot_dims, inv_freq=inv, positions=i32(pos.tolist()))
    close(y[..., :O], torch.einsum("nhi,hio->nho", x[..., :I], w.view(nh, I, O)), 1e-5, "product")
    close(y[..., O:], P.rotate_half(x[..., I:], pos, 1e4, rot_dims), 2e-4, "tail")


# ------------------------------------------------------------------------------------------ latent attention
def _case(T, H, dim, rd, vd, rank, q_rank, base, scale, seed, loud=None, sink=None):
    """A layer whose first projections pick columns of its input (so a test can set them) and whose W_o is the identity.
    ``loud`` = (query, key): the query's latent points along its last coordinate, which W_uq turns into a rotated part
    that meets the key's; no other query has that coordinate."""
    W = q_rank + rank + rd + H
    h = rnd(T, W, seed=seed)
    uq = rnd(H * (dim + rd), q_rank, seed=seed + 1, scale=q_rank ** -0.5)
    if loud is not None:
        qi, kj = loud
        half = rd // 2
        vec = torch.full((rd,), 2.0, dtype=F64)
        vec[0] = vec[half] = 0.0                                # the fastest pair turns too quickly to point anywhere
        h[kj, q_rank + rank:q_rank + rank + rd] = vec
        h[:, q_rank - 1] = 0.0
        h[qi, q_rank - 1] = 30.0
        uq.view(H, dim + rd, q_rank)[:, dim:, q_rank - 1] = vec
    eye = torch.eye(W, dtype=F64)
    p = {"dq": eye[:q_rank], "dq.norm": 1.0 + 0.2 * rnd(q_rank, seed=seed + 2), "uq": uq, "dkv": eye[q_rank:q_rank + rank + rd],
         "dkv.norm": 1.0 + 0.2 * rnd(rank, seed=seed + 3), "uk": rnd(H * dim, rank, seed=seed + 4, scale=rank ** -0.5),
         "uv": rnd(H * vd, rank, seed=seed + 5, scale=rank ** -0.5), "sink": rnd(H, seed=seed + 6) if sink is None else
         torch.full((H,), float(sink), dtype=F64), "g": eye[-H:], "o": torch.eye(H * vd, dtype=F64)}
    m = {"heads": H, "dim": dim, "rot_dim": rd, "vdim": vd, "kv_rank": rank, "q_rank": q_rank, "scale": scale}
    if rd:
        m["rot"] = {"dims": rd, "base": base}
    return h, p, m


def _part(m, p, dtype):
    from mivi_v4_b200.parts import PartSpec, build
    W = p["dq"].shape[1]
    pos = PartSpec("rope", dict(head_dim=m["rot_dim"], theta=m["rot"]["base"], style="half_split")) if m["rot_dim"] else PartSpec("none")
    part = build("mixer", PartSpec("latent_attention",
                                   dict(hidden=W, n_heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], value_dim=m["vdim"],
                                        kv_rank=m["kv_rank"], q_rank=m["q_rank"], scale=m["scale"], eps=1e-5, gated="head"),
                                   parts={"position": pos}))
    # (W_o takes the heads to vdim * heads columns here, not back to the width: the part never looks at its rows)
    vec = ("sink", "dq.norm", "dkv.norm")
    part.load({n: dev(v, torch.float32 if n in vec else dtype) for n, v in p.items()})
    return part


def _run(part, h_seqs, steps, dtype, page=16, splits=None, monkeypatch=None):
    """``h_seqs``: an input per sequence; ``steps``: lists of how many tokens each sequence brings in that step."""
    from mivi_v4_b200.cache import KVView
    k = K()
    if splits is not None:
        monkeypatch.setattr(k, "latent_splits", lambda *a: splits)
        monkeypatch.setattr(k, "latent_decode_splits", lambda *a: splits)
    per = [-(-x.shape[0] // page) for x in h_seqs]
    perm = torch.randperm(sum(per) + 3, generator=torch.Generator().manual_seed(5))[:sum(per)].tolist()      # pages in no order
    rows, at = [], 0
    for n in per:
        rows.append(perm[at:at + n] + [0] * (max(per) + 9 - n))
        at += n
    pool = torch.full((sum(per) + 3, page * (part.rank + part.rd)), float("nan"), dtype=dtype, device=DEV)
    done, outs = [0] * len(h_seqs), [[] for _ in h_seqs]
    for lens in steps:
        live = [b for b, n in enumerate(lens) if n]
        step = make_step([lens[b] for b in live], [done[b] for b in live], dtype, [rows[b] for b in live])
        view = KVView(pool, step.page_tables[0], page, True, part.cache_need())
        u = torch.cat([dev(h_seqs[b][done[b]:done[b] + lens[b]], dtype) for b in live])
        y = torch.full((u.shape[0], part.w_o.shape[0]), float("nan"), device=DEV)
        part.forward(u, y, step, view, accumulate=False)
        at = 0
        for b in live:
            outs[b].append(y[at:at + lens[b]])
            at += lens[b]
            done[b] += lens[b]
    k.check_device_errors()
    return [torch.cat(o) for o in outs]


SIZES = [(10, 8, 12, 6, 24, 20, 100.0, 8), (1, 20, 0, 20, 36, 9, 1.0, 16), (3, 5, 6, 10, 41, 33, 1e4, 8), (9, 32, 16, 48, 72, 64, 500.0, 64),
         (2, 64, 32, 64, 136, 24, 5e4, 16), (4, 8, 8, 16, 8, 16, 10.0, 32), (17, 16, 16, 16, 264, 40, 50.0, 16),
         (32, 64, 32, 64, 256, 96, 1e4, 64), (2, 128, 64, 128, 520, 16, 1e6, 64)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,dim,rd,vd,rank,q_rank,base,page", SIZES)
def test_latent_attention_with_a_query_latent_under_every_cut(dtype, H, dim, rd, vd, rank, q_rank, base, page):
    T = 150
    h, p, m = _case(T, H, dim, rd, vd, rank, q_rank, base, 0.3, seed=rank)
    if dtype == BF:
        h = h.to(dtype).double()
        p = {n: (v if n in ("sink", "dq.norm", "dkv.norm") else v.to(dtype).double()) for n, v in p.items()}
    want = P.latent_attention(h, p, m, 1e-5)
    part = _part(m, p, dtype)
    for cuts in ([T], [1] * T, [100] + [1] * 50, [2] * 75, [7] * 21 + [3], [63, 65, 22]):
        close(_run(part, [h], [[n] for n in cuts], dtype, page)[0], want, 5e-5 if dtype == torch.float32 else 2e-2, f"cuts {cuts[:3]}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("splits", [1, 2, 3, 7, 32])
@pytest.mark.parametrize("H,vd", [(2, 16), (11, 8)])
def test_keys_in_shares_and_batches_of_unequal_sequences(dtype, splits, H, vd, monkeypatch):
    """Single tokens whose keys are cut into shares (some without any key), several sequences in a step, each against
    itself alone; the sink counts once whatever the shares."""
    lens = (133, 40, 3)
    cases = [_case(T, H, 16, 8, vd, 40, 24, 1e3, 0.5, seed=3) for T in lens]
    p, m = cases[0][1], cases[0][2]
    hs = [rnd(T, p["dq"].shape[1], seed=50 + T) for T in lens]
    part = _part(m, p, dtype)
    steps = [[120, 30, 1]] + [[1, 1, 1]] * 2 + [[1, 1, 0]] * 8 + [[3, 0, 0]]
    got = _run(part, hs, steps, dtype, 16, splits, monkeypatch)
    for b, h in enumerate(hs):
        close(got[b], P.latent_attention(h, p, m, 1e-5), 5e-5 if dtype == torch.float32 else 2.5e-2, f"sequence {b}, {splits} shares")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("key", [0, 1, 15, 16, 17, 63, 64, 127, 128, 198, 199])
def test_a_loud_key_far_away_and_at_page_borders(dtype, key):
    """The last query and one key made to stand out among 200: the first keys, keys on both sides of page borders and
    of the kernels' key tiles, the query's own; in a whole prompt, in a prompt's later portion, decoded alone, with the
    keys in shares.  The row is decided by that key: losing it would show."""
    T, H, vd, rank = 200, 3, 16, 24
    h, p, m = _case(T, H, 16, 16, vd, rank, 16, 1e6, 0.5, seed=key, loud=(T - 1, key))
    want = P.latent_attention(h, p, m, 1e-5)
    alone = torch.sigmoid(h[T - 1, -H:])[:, None] * (P.latent_rows(h, p, m, 1e-5)[0][key] @ p["uv"].T).view(H, vd)
    assert (want[T - 1].view(H, vd) - alone).abs().max() < 0.05 * alone.abs().max()
    part = _part(m, p, dtype)
    tol = 5e-5 if dtype == torch.float32 else 2.5e-2
    for cuts in ([T], [T - 1, 1], [130, 70], [184, 16], [T - 2, 2], [190] + [1] * 10):
        got = _run(part, [h], [[n] for n in cuts], dtype)[0]
        close(got, want, tol, f"key {key} cuts {cuts[:3]}")
        close(got[T - 1], want[T - 1], tol, f"the loud row, key {key} cuts {cuts[:3]}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_sink_takes_its_share_in_every_kind_of_step(dtype):
    T = 80
    rows = {}
    for sink in (-30.0, 0.0, 4.0, 12.0):
        h, p, m = _case(T, 3, 16, 16, 16, 24, 16, 100.0, 0.4, seed=9, sink=sink)
        rows[sink] = P.latent_attention(h, p, m, 1e-5)
        part = _part(m, p, dtype)
        for cuts in ([T], [60] + [1] * 20, [1] * T):
            close(_run(part, [h], [[n] for n in cuts], dtype)[0], rows[sink], 5e-5 if dtype == torch.float32 else 2.5e-2, f"sink {sink}")
    assert rows[12.0].abs().median() < 0.02 * rows[-30.0].abs().median()


# ------------------------------------------------------------------------------------------ mixture of experts
@pytest.mark.parametrize("E,top", [(6, 2), (5, 1), (3, 3), (1, 1), (40, 6), (64, 32), (130, 4)])
def test_router_bias_and_softmax_over_the_chosen_logits(E, top):
    k = K()
    N = 57
    z = rnd(N, E, seed=E, scale=2.0).float().double()
    z[3] *= 100.0                                            # logits hundreds apart: nothing overflows, no ties from underflow
    b = rnd(E, seed=1).float().double()
    want = P.route(z + b, top)
    wide = torch.full((N, E + 9), float("nan"), dtype=F64)
    wide[:, :E] = z
    dense = torch.full((N, E), float("nan"), device=DEV)
    pick, pick_w = torch.zeros(N, top, dtype=torch.int32, device=DEV), torch.zeros(N, top, device=DEV)
    k.route(dev(wide)[:, :E], dense, pick, pick_w, E, 1, 1, top, False, mode=k.ROUTE_CHOSEN_SOFTMAX, bias=dev(b))
    close(dense, want, 1e-5, "dense weights")
    rows = torch.arange(N)[:, None].expand(N, top)
    close(pick_w, want[rows, pick.cpu().long()], 1e-5, "picked weights")
    assert (torch.sort(pick.cpu().long(), -1).values == torch.sort(torch.topk(z + b, top, -1).indices, -1).values).all()
    # the bias with the other scores: sigmoid and softmax of z + b
    k.route(dev(z), dense, pick, pick_w, E, 1, 1, top, False, mode=k.ROUTE_SOFTMAX, bias=dev(b))
    s = torch.softmax(z + b, -1)
    w = torch.gather(s, 1, pick.cpu().long())
    close(pick_w, w / w.sum(-1, keepdim=True), 1e-5, "softmax with a bias")


def _clamped(g, u, limit, alpha=1.702):
    g, u = g.clamp(max=limit), u.clamp(-limit, limit)
    return g * torch.sigmoid(alpha * g) * (u + 1.0)


def grouped(wg, wu, G=16):
    F, H = wg.shape
    return torch.stack([wg.view(F // G, G, H), wu.view(F // G, G, H)], dim=1).reshape(2 * F, H).contiguous()


@pytest.mark.parametrize("group", [0, 4, 16])
@pytest.mark.parametrize("out_dtype", DTYPES)
def test_clamped_activation_of_alternating_columns(out_dtype, group):
    k = K()
    N, F = 7, 48
    g, u = rnd(N, F, scale=2.0), rnd(N, F, seed=1, scale=2.0)
    gu = torch.cat([g, u], 1) if not group else \
        torch.stack([g.view(N, F // group, group), u.view(N, F // group, group)], 2).reshape(N, 2 * F)
    out = torch.full((N, F), float("nan"), dtype=out_dtype, device=DEV)
    k.glu_clamped(dev(gu), out, 1.1, 1.702, group)
    close(out, _clamped(g, u, 1.1), 2e-6 if out_dtype == torch.float32 else 5e-3)


@pytest.mark.parametrize("M", [1, 8, 9, 33, 64, 65, 200, 1000])
@pytest.mark.parametrize("F1,F2,Kd", [(16, 16, 8), (48, 16, 72), (256, 128, 96), (4096, 1024, 520), (1040, 0, 200)])
def test_products_that_apply_the_clamped_activation(M, F1, F2, Kd):
    """Two runs of features with limits of their own in one matrix, in every kernel that takes the shape."""
    k = K()
    F = F1 + F2
    x = rnd(M, Kd).to(BF).to(DEV)
    wg, wu = rnd(F, Kd, seed=1, scale=2.0 * Kd ** -0.5).to(BF).to(DEV), rnd(F, Kd, seed=2, scale=2.0 * Kd ** -0.5).to(BF).to(DEV)
    a, b = x.double() @ wg.double().T, x.double() @ wu.double().T
    want = torch.cat([_clamped(a[:, :F1], b[:, :F1], 0.6), _clamped(a[:, F1:], b[:, F1:], 1.7)], 1).cpu()
    limits = k.glu_limits([(F1, 0.6), (F2, 1.7)], 1.702, DEV)
    many = [functools.partial(k.gemm_tc, pair=False), k.gemm_tc_swap] + \
        ([functools.partial(k.gemm_tc, pair=True)] if M > 128 and 2 * F >= 128 else [])
    for fn in ([k.gemm_small_m, k.gemm_tc_swap] if M <= 64 else many):
        out = torch.full((M, F), float("nan"), dtype=BF, device=DEV)
        fn(x, grouped(wg, wu), out, swiglu=True, limits=limits)
        k.check_device_errors()
        close(out, want, 1e-2, str(fn))


def _moe_case(H, mlp, seed):
    r = mlp["router"]
    E, ff = r["experts"], mlp["expert"]["ff"]
    u = rnd(H, seed=seed)
    u = u / u.norm()
    p = {"router": (torch.linspace(-1.5, 2.5, E, dtype=F64)[torch.randperm(E, generator=torch.Generator().manual_seed(seed))])[:, None] * u,
         "router.b": 0.1 * rnd(E, seed=seed + 1)}
    for e, f in [(f"e{i}.", ff) for i in range(E)] + ([("shared.", mlp["shared"]["ff"])] if mlp.get("shared") else []):
        n = len(p)
        p.update({e + "gate": rnd(f, H, seed=n, scale=1.5 * H ** -0.5), e + "up": rnd(f, H, seed=n + 1, scale=1.5 * H ** -0.5),
                  e + "down": rnd(H, f, seed=n + 2, scale=f ** -0.5)})
    return p, u


MIXTURES = [(64, dict(kind="moe", expert=dict(ff=32, limit=0.9), shared=dict(ff=48, limit=1.6), router=dict(experts=6, top=2))),
            (40, dict(kind="moe", expert=dict(ff=16, limit=1.2), router=dict(experts=3, top=1))),
            (72, dict(kind="moe", expert=dict(ff=20, limit=0.7), shared=dict(ff=10, limit=0.4), router=dict(experts=5, top=5))),
            (128, dict(kind="moe", expert=dict(ff=64, limit=7.0), shared=dict(ff=20, limit=1.0), router=dict(experts=8, top=4))),
            (51, dict(kind="moe", expert=dict(ff=32, limit=0.8), shared=dict(ff=16, limit=0.9), router=dict(experts=2, top=1)))]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,mlp", MIXTURES)
def test_mixture_in_short_long_and_sorted_steps(H, mlp, dtype, monkeypatch):
    """Few rows, more rows than the gated products start from, and rows sorted by expert; with the residual gate's rows
    riding in the router's product."""
    from mivi_v4_b200.parts import PartSpec, build
    from mivi_v4_b200.parts.feed_forward import RoutedExperts
    p, u = _moe_case(H, mlp, seed=H)
    r, sh = mlp["router"], mlp.get("shared") or {}
    side = rnd(H, H, seed=77, scale=H ** -0.5)
    if dtype == BF:
        p = {n: (v if n == "router.b" else v.to(BF).double()) for n, v in p.items()}
        side = side.to(BF).double()
    for lowered in (False, True):
        if lowered:
            monkeypatch.setattr(RoutedExperts, "SORTED_ROWS_AN_EXPERT", 1)
        part = build("feed_forward", PartSpec("routed_experts", dict(
            hidden=H, n_experts=r["experts"], ff=mlp["expert"]["ff"], top=r["top"], score="chosen_softmax", router_bias=True,
            shared_ff=sh.get("ff", 0), shared_gate=False, act="clamped", limit=mlp["expert"]["limit"], shared_limit=sh.get("limit", 0.0))))
        part.load({n: dev(v, torch.float32 if n == "router.b" else dtype) for n, v in p.items()})
        assert part.take_side_rows(dev(side, dtype))
        for N in (1, 8, 50, 70, 300):
            h = rnd(N, H, seed=N)
            h = h - (h @ u)[:, None] * u + torch.where(torch.arange(N) % 3 == 0, 3.0, -2.5)[:, None].double() * u    # no close calls
            h = h.to(dtype).double()
            step = make_step([N], [0], dtype, [[0]])
            y = torch.full((N, H), float("nan"), device=DEV)
            part.forward(dev(h, dtype), y, step, accumulate=False)
            K().check_device_errors()
            close(y, P.moe(h, p, mlp), 2e-5 if dtype == torch.float32 else 1.5e-2, f"{N} rows, sorted {lowered}")
            close(part.side, h @ side.T, 1e-5, "side rows")
            part.forward(dev(h, dtype), y, step)                       # and added to what is there
            close(y, 2.0 * P.moe(h, p, mlp), 2e-5 if dtype == torch.float32 else 1.5e-2, f"{N} rows twice, sorted {lowered}")


# ------------------------------------------------------------------------------------------ embedding
def test_bigram_embedding_writes_rounded_rows():
    k = K()
    V, H, buckets = 50, 24, 13
    table, bigram = rnd(V, H), rnd(buckets + 1, H, seed=1)
    toks = torch.randint(0, V, (30,), generator=torch.Generator().manual_seed(3)).tolist()
    cfg = {"embedding": {"bigram": {"buckets": buckets, "mul_prev": 5, "mul_cur": 3}}}
    for dtype in DTYPES:
        prev = torch.zeros(2, dtype=torch.int32, device=DEV)
        out = torch.full((30, H), float("nan"), device=DEV)
        rounded = torch.full((30, H), float("nan"), dtype=BF, device=DEV)
        k.embed_bigram(dev(table, dtype), dev(bigram, dtype), i32(toks), i32(list(range(30))), i32([0] * 30), i32([0, 30]), i32([1]), prev,
                       out, None, 5, 3, rounded=rounded)
        close(out, P.embedding(toks, table.to(dtype), bigram.to(dtype), cfg), 1e-6)
        assert torch.equal(rounded, out.to(BF)) and prev.tolist() == [0, toks[-1]]
