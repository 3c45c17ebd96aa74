"""Every kernel that the Mevulix decoder added or widened, alone, against the plain implementation's function of the
same mechanism (float64), at sizes of the tests' own: the layer norm on a sublayer's output, q prepared with biases, whole
norms and a temperature (with and without keys and values of its own), attention with a table of distances under every
cut, loud keys at the buckets' edges, at page borders and far away, latent attention with neighbouring pairs and stretched
frequencies, gelu and experts' weights inside every matrix product, the router without renormalization, the mixture whose
weights multiply its inputs in short, long and sorted steps."""
import functools

import pytest
import torch

import plain_mevulix as P

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
@pytest.mark.parametrize("H,N", [(24, 3), (50, 5), (516, 9), (2048, 2), (4096, 3), (5000, 2), (8, 1), (1, 2)])
def test_layer_norm_on_a_sublayers_output_joins_the_stream(H, N):
    k = K()
    x, y, y2 = rnd(N, H), 3.0 + rnd(N, H, seed=1), rnd(N, H, seed=2)
    w, b = 1 + rnd(H, seed=5), rnd(H, seed=6)
    for two in (False, True):
        v = 1.5 * y + (-0.5 * y2 if two else 0.0)
        for centered in (True, False):
            want = x + (P.layer_norm(v, w, b, 1e-3) if centered else P.rms_norm(v, w, 1e-3))
            for dtype in (None, torch.float32, BF):
                resid = dev(x)
                rounded = None if dtype is None else torch.full((N, H), float("nan"), dtype=dtype, device=DEV)
                k.norm_add_sum(dev(y), dev(w), 1e-3, resid, bias=dev(b) if centered else None, s1=1.5, y2=dev(y2) if two else None,
                               s2=-0.5, rounded=rounded)
                close(resid, want, 1e-5, f"centered {centered}, two branches {two}")
                if rounded is not None:
                    assert torch.equal(rounded, resid.to(dtype))


def test_final_norm_with_a_gain():
    from mivi_v4_b200.parts import PartSpec, build
    n = build("norm", PartSpec("layernorm", dict(dim=200, eps=1e-2, bias=True, gain=2.5)))
    w, b, x = 1 + rnd(200, seed=1), rnd(200, seed=2), rnd(5, 200)
    n.load({"weight": dev(w), "bias": dev(b)})
    out = torch.empty(2, 200, device=DEV)
    n.forward(dev(x), out, rows=i32([3, 1]))
    close(out, 2.5 * P.layer_norm(x, w, b, 1e-2)[[3, 1]], 3e-6)


# ------------------------------------------------------------------------------------------ attention
def _att_case(T, m, rows, seed, loud=None, sink=None):
    """A layer whose first projections pick columns of its input (so a test can set them) and whose W_o is the identity.
    ``loud`` = (query, key): in the space that the norms leave, the query's and the key's heads point the same way."""
    H, G, dk, dv = (m[n] for n in ("heads", "kv_heads", "dim", "vdim"))
    nq, nk, nv = H * dk, G * dk, G * dv
    W = nq + nk + nv
    h = rnd(T, W, seed=seed)
    p = {"q.b": 0.3 * rnd(nq, seed=seed + 1), "k.b": 0.3 * rnd(nk, seed=seed + 2), "v.b": rnd(nv, seed=seed + 3),
         "q.norm": 1 + 0.2 * rnd(nq, seed=seed + 4), "k.norm": 1 + 0.2 * rnd(nk, seed=seed + 5),
         "rel": 1.5 * rnd(rows, H, seed=seed + 6), "sink": rnd(H, seed=seed + 7) if sink is None else torch.full((H,), float(sink), dtype=F64),
         "o": torch.eye(H * dv, dtype=F64)}
    if loud is not None:
        i, j = loud
        h[:, nq] = 0.0                                          # no other key has the first element of kv head 0
        p["k.b"][0] = 0.0
        h[j, nq:nq + nk] = 0.0
        h[j, nq] = 50.0
        h[i, :nq] = 0.0
        h[i, 0:nq:dk] = 50.0
    eye = torch.eye(W, dtype=F64)
    p.update({"q": eye[:nq], "k": eye[nq:nq + nk], "v": eye[nq + nk:]})
    return h, p


VEC = ("q.b", "k.b", "v.b", "q.norm", "k.norm", "rel", "sink")


def _att_part(m, p, dtype, shared=False):
    from mivi_v4_b200.parts import PartSpec, build
    part = build("mixer", PartSpec("sink_attention", dict(
        hidden=p["q"].shape[1], n_heads=m["heads"], n_kv_heads=m["kv_heads"], key_dim=m["dim"], value_dim=m["vdim"], scale=m["scale"],
        softcap=m["softcap"], qk_norm_eps=1e-5, sink=True, gated=False, split_weights=True, proj_bias=True,
        q_temp=(m["q_temp"]["coef"], m["q_temp"]["every"]), bias_max=m["bias_max"], bias_rows=p["rel"].shape[0], shared_kv=shared),
        parts={"position": PartSpec("none")}))
    part.load({n: dev(p[n], torch.float32 if n in VEC else dtype) for n in part.param_specs()})
    return part


def _pages(lens, page):
    per = [-(-n // page) for n in lens]
    perm = torch.randperm(sum(per) + 3, generator=torch.Generator().manual_seed(5))[:sum(per)].tolist()      # pages in no order
    rows, at = [], 0
    for n in per:
        rows.append(perm[at:at + n] + [0] * (max(per) + 2 - n))
        at += n
    return rows, sum(per) + 3


def _run(part, h_seqs, steps, dtype, page=16, reader=None, reader_seqs=None):
    """``h_seqs``: an input per sequence; ``steps``: lists of how many tokens each sequence brings in that step.  With
    ``reader`` that part runs after ``part`` in every step, on ``reader_seqs``, from the cache that ``part`` fills; its
    results come back instead."""
    from mivi_v4_b200.cache import KVView
    rows, n_pages = _pages([x.shape[0] for x in h_seqs], page)
    need = part.cache_need()
    shape = (n_pages, need.page_elements(page)) if need.uneven else (n_pages, 2, need.n_kv_heads, page, need.head_dim)
    pool = torch.full(shape, float("nan"), dtype=dtype, device=DEV)
    done, outs = [0] * len(h_seqs), [[] for _ in h_seqs]
    for lens in steps:
        live = [b for b, n in enumerate(lens) if n]
        step = make_step([lens[b] for b in live], [done[b] for b in live], dtype, [rows[b] for b in live])
        for who, seqs, writable in ((part, h_seqs, True),) + (((reader, reader_seqs, False),) if reader is not None else ()):
            u = torch.cat([dev(seqs[b][done[b]:done[b] + lens[b]], dtype) for b in live])
            y = torch.full((u.shape[0], who.w_o.shape[0]), float("nan"), device=DEV)
            who.forward(u, y, step, KVView(pool, step.page_tables[0], page, writable, need), accumulate=False)
        at = 0
        for b in live:
            outs[b].append(y[at:at + lens[b]])
            at += lens[b]
            done[b] += lens[b]
    K().check_device_errors()
    return [torch.cat(o) for o in outs]


def _m(H, G, dk, dv, scale, cap, coef, every, reach):
    return {"heads": H, "kv_heads": G, "dim": dk, "vdim": dv, "scale": scale, "softcap": cap, "q_temp": {"coef": coef, "every": every},
            "bias_max": reach}


def _rounded(h, p, dtype):
    if dtype == BF:
        h = h.to(BF).double()
        p = {n: (v if n in VEC else v.to(BF).double()) for n, v in p.items()}
    return h, p


ATT = [(_m(6, 2, 32, 16, 0.4, 5.0, 0.8, 7, 40), 12, 16), (_m(1, 1, 8, 8, 1.0, 30.0, 0.5, 1, 64), 8, 64),
       (_m(3, 1, 11, 9, 0.5, 2.0, 1.5, 50, 20), 2, 8), (_m(4, 4, 16, 128, 0.7, 8.0, 0.3, 33, 2000), 31, 16),
       (_m(8, 1, 64, 48, 0.3, 20.0, 0.4, 64, 33), 9, 32), (_m(10, 5, 128, 64, 0.2, 9.0, 0.1, 100, 110), 16, 64),
       (_m(2, 2, 250, 256, 0.2, 4.0, 0.6, 10, 7), 3, 16), (_m(12, 1, 48, 32, 0.4, 6.0, 0.2, 30, 90), 20, 16),
       (_m(40, 2, 16, 16, 0.5, 5.0, 0.4, 25, 50), 6, 8), (_m(5, 5, 256, 256, 0.1, 9.0, 0.3, 12, 30), 10, 16)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m,rows,page", ATT)
def test_attention_with_a_bias_by_distance_under_every_cut(m, rows, page, dtype):
    T = 150
    h, p = _rounded(*_att_case(T, m, rows, seed=rows), dtype)
    want = P.attention(h, p, m, 1e-5)[0]
    part = _att_part(m, p, dtype)
    for cuts in ([T], [1] * T, [100] + [1] * 50, [2] * 75, [7] * 21 + [3], [63, 65, 22]):
        close(_run(part, [h], [[n] for n in cuts], dtype, page)[0], want, 5e-5 if dtype == torch.float32 else 2e-2, f"cuts {cuts[:3]}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m,rows,page", [ATT[0], ATT[2], ATT[4]])
def test_a_layer_that_reads_another_layers_keys_and_values(m, rows, page, dtype):
    """Its own queries, temperature, cap, bias and sink, the other layer's keys and values; batches of unequal
    sequences, each against itself alone."""
    lens = (133, 40, 3)
    _, p = _att_case(8, m, rows, seed=1)
    m2 = dict(m, scale=1.3 * m["scale"], softcap=0.7 * m["softcap"], q_temp={"coef": 0.9, "every": 11}, bias_max=m["bias_max"] + 9)
    _, p2 = _att_case(8, m2, rows + 3, seed=40)
    hs, hs2 = [rnd(T, p["q"].shape[1], seed=50 + T) for T in lens], [rnd(T, p["q"].shape[1], seed=90 + T) for T in lens]
    if dtype == BF:
        hs, hs2 = [h.to(BF).double() for h in hs], [h.to(BF).double() for h in hs2]
    part, reader = _att_part(m, p, dtype), _att_part(m2, p2, dtype, shared=True)
    assert not hasattr(reader, "k_b") and reader.w_qkvg.shape[0] < part.w_qkvg.shape[0]
    steps = [[120, 30, 1]] + [[1, 1, 1]] * 2 + [[1, 1, 0]] * 8 + [[3, 0, 0]]
    got = _run(part, hs, steps, dtype, page, reader, hs2)
    for b in range(3):
        kv = P.keys_and_values(hs[b], p, m, 1e-5)
        close(got[b], P.attention(hs2[b], p2, m2, 1e-5, kv=kv)[0], 5e-5 if dtype == torch.float32 else 2.5e-2, f"sequence {b}")
    with pytest.raises(RuntimeError):
        _run(reader, hs2, [[4, 4, 3]], dtype, page)


# with 12 rows that reach 40 the rows start at distances 0 .. 6 and 9, 12, 16, 22, 30; 39 and 40 lie in the last one
EDGES = [0, 5, 6, 8, 9, 11, 12, 15, 16, 21, 22, 29, 30, 39, 40, 47, 48, 63, 64, 127, 128, 198, 199]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("back", EDGES)
def test_a_loud_key_at_every_edge_of_the_buckets_and_far_away(back, dtype):
    """The last query and the key ``back`` tokens before it, made to stand out among 200, and a bias that changes by 6
    from bucket to bucket: the row's weights depend on the bucket of that distance, in a whole prompt, in a later portion,
    decoded alone, in portions down to two tokens."""
    T = 200
    m = _m(4, 2, 16, 16, 1.0, 6.0, 0.2, 9, 40)
    h, p = _att_case(T, m, 12, seed=back, loud=(T - 1, T - 1 - back), sink=1.0)
    p["rel"] = torch.where(torch.arange(12) % 2 == 0, 3.0, -3.0)[:, None].double() * torch.ones(1, 4, dtype=F64) + 0.1 * rnd(12, 4)
    h, p = _rounded(h, p, dtype)
    want = P.attention(h, p, m, 1e-5)[0]
    # one bucket off would show
    moved = dict(m)
    for reach in (40 / 1.25, 40 * 1.25):
        moved["bias_max"] = reach
        off = (P.attention(h, p, moved, 1e-5)[0][T - 1] - want[T - 1]).abs().max() / want[T - 1].abs().max()
        assert back < 6 or back >= 40 or off > 0.05 or P.bucket(back, 12, reach) == P.bucket(back, 12, 40), (back, off)
    part = _att_part(m, p, dtype)
    tol = 5e-5 if dtype == torch.float32 else 2.5e-2
    for cuts in ([T], [T - 1, 1], [130, 70], [184, 16], [T - 2, 2], [190] + [1] * 10):
        got = _run(part, [h], [[n] for n in cuts], dtype)[0]
        close(got, want, tol, f"{back} back, cuts {cuts[:3]}")
        close(got[T - 1], want[T - 1], tol, f"the loud row, {back} back, cuts {cuts[:3]}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_distance_table_longer_than_shared_memory_holds_and_of_one_number(dtype):
    """Tables of 1, 2, 65, 2,048 and 2,049 distances, with keys on both sides of the table's end."""
    k = K()
    H, G, dk, dv, T, ps = 3, 1, 32, 32, 2300, 64
    q, key, v = rnd(T, H, dk), rnd(T, G, dk, seed=1), rnd(T, G, dv, seed=2)
    q, key, v = (x.to(dtype).double() for x in (q, key, v))
    rows, n_pages = _pages([T], ps)
    pool = torch.zeros(n_pages, 2, G, ps, dk, dtype=dtype, device=DEV)
    for blk, page in enumerate(rows[0][:-(-T // ps)]):
        n = min(ps, T - blk * ps)
        pool[page, 0, :, :n] = dev(key[blk * ps:blk * ps + n].permute(1, 0, 2), dtype)
        pool[page, 1, :, :n] = dev(v[blk * ps:blk * ps + n].permute(1, 0, 2), dtype)
    places = [0, 1, 63, 64, 65, 66, 700, 2046, 2047, 2048, 2049, 2100, T - 1]
    for L in (1, 2, 65, 2048, 2049):
        table = rnd(H, L, seed=L)
        s = torch.einsum("thd,shd->hts", q[places], key.expand(T, H, dk)) * 0.2
        s = 4.0 * torch.tanh(s / 4.0)
        back = torch.tensor(places)[:, None] - torch.arange(T)[None, :]
        s = (s + table[:, back.clamp(0, L - 1)]).masked_fill(back[None] < 0, float("-inf"))
        want = torch.einsum("hts,shd->thd", torch.softmax(s, -1), v.expand(T, H, dv)).reshape(len(places), -1)
        out = torch.full((len(places), H * dv), float("nan"), dtype=dtype, device=DEV)
        for tile in (0, 1, 2, 4):
            k.attention_sink(dev(q[places].reshape(-1, H * dk), dtype), pool, ps, i32([rows[0]]), i32(places), i32([0] * len(places)), out,
                             H, G, dk, dv, 0.2, softcap=4.0, distance_table=dev(table), head_tile=tile)
            close(out, want, 2e-5 if dtype == torch.float32 else 1.5e-2, f"{L} distances, {tile} heads a block")
        if dtype == BF:
            full = torch.full((T, H * dv), float("nan"), dtype=dtype, device=DEV)
            k.attention_sink_prefill(dev(q.reshape(T, -1), dtype), pool, ps, i32([rows[0]]), i32([0, T]), i32([0]), full, 1, H, G, dk, dv,
                                     0.2, softcap=4.0, distance_table=dev(table), split_weights=True)
            close(full[places], want, 1.5e-2, f"{L} distances on the tensor cores")
            for splits in (1, 5):
                part = (torch.empty(len(places), H, splits, dv, device=DEV), torch.empty(len(places), H, splits, 2, device=DEV))
                k.attention_sink_decode(dev(q[places].reshape(-1, H * dk), dtype), pool, ps, i32([rows[0]]), i32(places), i32([0] * len(places)),
                                        out, H, G, dk, dv, 0.2, softcap=4.0, distance_table=dev(table), splits=splits, part=part)
                close(out, want, 1.5e-2, f"{L} distances, single tokens on the tensor cores, {splits} shares")


@pytest.mark.parametrize("splits", [1, 2, 3, 7, 32])
@pytest.mark.parametrize("H,G,dk,dv", [(4, 2, 64, 64), (9, 1, 32, 48), (20, 1, 16, 16), (8, 8, 128, 96), (3, 1, 80, 160), (2, 2, 240, 256)])
def test_single_tokens_on_the_tensor_cores_windows_chunks_caps_sinks_and_shares(H, G, dk, dv, splits):
    """Tokens at many places of two sequences, their keys in shares (some without any key), with a window or a chunked mask,
    a key that stands out just inside and just outside, with and without a cap, a sink and a table."""
    k = K()
    T, ps = 230, 16
    places, seqs = [0, 1, 15, 16, 17, 63, 64, 65, 99, 127, 128, 200, T - 1, 5, 77, 150], [0] * 13 + [1] * 3
    key, v = rnd(2, T, G, dk).to(BF).double(), rnd(2, T, G, dv, seed=1).to(BF).double()
    rows, n_pages = _pages([T, T], ps)
    pool = torch.zeros(n_pages, G * ps * (dk + dv), dtype=BF, device=DEV)
    for b in range(2):
        for blk, page in enumerate(rows[b][:-(-T // ps)]):
            n = min(ps, T - blk * ps)
            pool[page, :G * ps * dk].view(G, ps, dk)[:, :n] = dev(key[b, blk * ps:blk * ps + n].permute(1, 0, 2), BF)
            pool[page, G * ps * dk:].view(G, ps, dv)[:, :n] = dev(v[b, blk * ps:blk * ps + n].permute(1, 0, 2), BF)
    if dk == dv:
        pool = pool.view(n_pages, 2, G, ps, dk)
    part = (torch.full((16, H, splits, dv), float("nan"), device=DEV), torch.full((16, H, splits, 2), float("nan"), device=DEV))
    table, sink = rnd(H, 70, seed=4), rnd(H, seed=5)
    for window, chunk, cap, with_sink, with_table in ((0, 0, 5.0, True, True), (64, 0, 0.0, True, False), (65, 0, 3.0, False, True),
                                                      (0, 48, 0.0, False, False), (1, 0, 0.0, True, True), (0, 64, 9.0, True, False)):
        q = rnd(16, H, dk, seed=2)
        for n, (p, b) in enumerate(zip(places, seqs)):         # one key stands out: the first one seen, or the last one not seen
            lo = max(0, p - window + 1) if window else (p - p % chunk if chunk else 0)
            j = max(lo - n % 2, 0)
            q[n] = q[n] + 3.0 * key[b, j].repeat_interleave(H // G, dim=0)
        q = q.to(BF).double()
        s = torch.einsum("nhd,nshd->nhs", q, torch.stack([key[b] for b in seqs]).repeat_interleave(H // G, dim=2)) * dk ** -0.5
        s = cap * torch.tanh(s / cap) if cap else s
        back = torch.tensor(places)[:, None] - torch.arange(T)[None, :]
        if with_table:
            s = s + table[:, back.clamp(0, 69)].permute(1, 0, 2)
        gone = back < 0
        if window:
            gone = gone | (back >= window)
        if chunk:
            gone = gone | (torch.arange(T)[None, :] // chunk != torch.tensor(places)[:, None] // chunk)
        s = s.masked_fill(gone[:, None, :], float("-inf"))
        if with_sink:
            s = torch.cat([s, sink[None, :, None].expand(16, H, 1)], -1)
        w = torch.softmax(s, -1)[..., :T]
        want = torch.einsum("nhs,nshd->nhd", w, torch.stack([v[b] for b in seqs]).repeat_interleave(H // G, dim=2)).reshape(16, -1)
        out = torch.full((16, H * dv), float("nan"), dtype=BF, device=DEV)
        k.attention_sink_decode(dev(q.reshape(16, -1), BF), pool, ps, i32(rows), i32(places), i32(seqs), out, H, G, dk, dv, dk ** -0.5,
                                softcap=cap, window=window, chunk=chunk, sinks=dev(sink) if with_sink else None,
                                distance_table=dev(table) if with_table else None, splits=splits, part=part)
        close(out, want, 6e-3, f"window {window} chunk {chunk} cap {cap}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_query_temperature_changes_exactly_at_its_steps(dtype):
    """q alone, at the last token before and the first token of several steps, with and without a norm."""
    k = K()
    H, dk = 3, 20
    places = [0, 1, 5, 6, 7, 12, 13, 14, 99, 127, 128, 6999, 7000, 69998, 69999, 100000]
    N = len(places)
    proj, w = rnd(N, H * dk + 4), 1 + 0.3 * rnd(H * dk, seed=1)
    pool = torch.zeros(1, 2, 1, 16, dk, dtype=dtype, device=DEV)
    for every, coef in ((7, 0.5), (1, 0.2), (128, -0.1), (7000, 3.0)):
        grow = P.temperature(torch.tensor(places), {"coef": coef, "every": every})[:, None]
        for wq in (None, w):
            want = grow * (proj[:, :H * dk] if wq is None else P.rms_norm(proj[:, :H * dk], wq, 1e-4))
            q = torch.full((N, H * dk), float("nan"), dtype=dtype, device=DEV)
            k.qkv_prepare_wide(dev(proj), None if wq is None else dev(wq), None, 1e-4, 0, None, i32(places), i32([0] * N), i32([[0]]),
                               pool, 16, q, H, 0, dk, dk, q_temp=(coef, every))
            close(q / dev(grow).to(dtype), want / grow, 3e-6 if dtype == torch.float32 else 1.2e-2, f"every {every}")
    assert not pool.any()


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_sink_takes_its_share_and_is_neither_capped_nor_biased(dtype):
    T, m = 80, _m(3, 1, 16, 16, 0.5, 2.0, 0.3, 20, 20)
    rows = {}
    for sink in (-30.0, 0.0, 4.0, 12.0):                      # (12: six times the cap)
        h, p = _rounded(*_att_case(T, m, 6, seed=9, sink=sink), dtype)
        rows[sink] = P.attention(h, p, m, 1e-5)[0]
        part = _att_part(m, p, dtype)
        for cuts in ([T], [60] + [1] * 20, [1] * T):
            close(_run(part, [h], [[n] for n in cuts], dtype)[0], rows[sink], 5e-5 if dtype == torch.float32 else 2.5e-2, f"sink {sink}")
    assert rows[12.0].abs().median() < 0.05 * rows[-30.0].abs().median()


# ------------------------------------------------------------------------------------------ latent attention
def _lat_case(T, m, seed, loud=None):
    """As above for latent attention.  ``loud`` = (query, key): the query's latent points along its last coordinate, which
    W_uq turns into a rotated part that meets the key's; no other query has that coordinate."""
    H, dim, rd, vd, rank, q_rank = (m[n] for n in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank"))
    W = q_rank + rank + rd
    h = rnd(T, W, seed=seed)
    uq = rnd(H * (dim + rd), q_rank, seed=seed + 1, scale=q_rank ** -0.5)
    if loud is not None:
        qi, kj = loud
        vec = torch.full((rd,), 2.0, dtype=F64)
        vec[:2] = 0.0                                           # the fastest pair turns too quickly to point anywhere
        h[kj, q_rank + rank:] = vec
        h[:, q_rank - 1] = 0.0
        h[qi, q_rank - 1] = 30.0
        uq.view(H, dim + rd, q_rank)[:, dim:, q_rank - 1] = vec
    eye = torch.eye(W, dtype=F64)
    p = {"dq": eye[:q_rank], "dq.norm": 1.0 + 0.2 * rnd(q_rank, seed=seed + 2), "uq": uq, "dkv": eye[q_rank:],
         "dkv.norm": 1.0 + 0.2 * rnd(rank, seed=seed + 3), "uk": rnd(H * dim, rank, seed=seed + 4, scale=rank ** -0.5),
         "uv": rnd(H * vd, rank, seed=seed + 5, scale=rank ** -0.5), "o": torch.eye(H * vd, dtype=F64)}
    return h, p


def _lat_part(m, p, dtype):
    from mivi_v4_b200.parts import PartSpec, build
    pos = PartSpec("none")
    if m["rot_dim"]:
        rot = dict(head_dim=m["rot_dim"], theta=m["rot"]["base"], style="interleaved")
        s = m["rot"].get("scaling")
        pos = PartSpec("rope_yarn", dict(rot, **s)) if s else PartSpec("rope", rot)
    part = build("mixer", PartSpec("latent_attention", dict(
        hidden=p["dq"].shape[1], n_heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], value_dim=m["vdim"], kv_rank=m["kv_rank"],
        q_rank=m["q_rank"], scale=m["scale"], eps=1e-5, sink=False, gated=False), parts={"position": pos}))
    part.load({n: dev(v, torch.float32 if n.endswith(".norm") else dtype) for n, v in p.items()})
    return part


def _lm(heads, dim, rd, vd, rank, q_rank, base, scale, scaling=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rd, "vdim": vd, "kv_rank": rank, "q_rank": q_rank, "scale": scale}
    if rd:
        m["rot"] = {"dims": rd, "base": base}
        if scaling:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return m


def _round_lat(h, p, dtype):
    if dtype == BF:
        h, p = h.to(BF).double(), {n: (v if n.endswith(".norm") else v.to(BF).double()) for n, v in p.items()}
    return h, p


LAT = [(_lm(10, 8, 12, 6, 24, 20, 100.0, 0.3, (4.0, 64, 8.0, 1.0)), 8), (_lm(1, 20, 0, 20, 36, 9, 1.0, 0.3), 16),
       (_lm(3, 5, 6, 10, 41, 33, 1e4, 0.3), 8), (_lm(9, 32, 16, 48, 72, 64, 500.0, 0.3, (16.0, 100, 32.0, 1.0)), 64),
       (_lm(2, 64, 32, 64, 136, 24, 5e4, 0.1, (2.0, 4096, 32.0, 1.0)), 16), (_lm(4, 8, 8, 16, 8, 16, 10.0, 0.5, (40.0, 16, 2.0, 0.5)), 32),
       (_lm(32, 64, 32, 64, 256, 96, 1e4, 0.1, (8.0, 128, 16.0, 2.0)), 64), (_lm(2, 128, 64, 128, 520, 16, 1e6, 0.1, (3.0, 700, 20.0, 1.0)), 64)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m,page", LAT)
def test_latent_attention_with_neighbouring_pairs_and_stretched_frequencies(m, page, dtype):
    T = 150
    h, p = _round_lat(*_lat_case(T, m, seed=m["kv_rank"]), dtype)
    want = P.latent_attention(h, p, m, 1e-5)
    part = _lat_part(m, p, dtype)
    for cuts in ([T], [1] * T, [100] + [1] * 50, [2] * 75, [7] * 21 + [3], [63, 65, 22]):
        close(_run(part, [h], [[n] for n in cuts], dtype, page)[0], want, 5e-5 if dtype == torch.float32 else 2e-2, f"cuts {cuts[:3]}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("key", [0, 1, 15, 16, 63, 64, 127, 128, 198, 199])
def test_a_loud_latent_key_far_away_and_at_page_borders(dtype, key):
    """A row decided by one key whose rotated part meets the query's: a pair turned the wrong way, a factor left off or a
    lost key would show."""
    T = 200
    m = _lm(3, 16, 16, 16, 24, 16, 1e6, 0.5, (8.0, 1000, 4.0, 1.0))
    h, p = _round_lat(*_lat_case(T, m, seed=key, loud=(T - 1, key)), dtype)
    want = P.latent_attention(h, p, m, 1e-5)
    alone = (P.latent_rows(h, p, m, 1e-5)[0][key] @ p["uv"].T).view(3, 16)
    assert (want[T - 1].view(3, 16) - alone).abs().max() < 0.05 * alone.abs().max()
    part = _lat_part(m, p, dtype)
    tol = 5e-5 if dtype == torch.float32 else 2.5e-2
    for cuts in ([T], [T - 1, 1], [130, 70], [184, 16], [T - 2, 2], [190] + [1] * 10):
        got = _run(part, [h], [[n] for n in cuts], dtype)[0]
        close(got, want, tol, f"key {key} cuts {cuts[:3]}")
        close(got[T - 1], want[T - 1], tol, f"the loud row, key {key} cuts {cuts[:3]}")


@pytest.mark.parametrize("N", [3, 8, 70])
@pytest.mark.parametrize("nh,I,O,rot,rot_dims", [(3, 16, 24, 8, 8), (2, 5, 70, 6, 4), (1, 64, 130, 34, 34)])
def test_the_queries_tails_and_the_long_steps_queries_grow_with_the_rotation(nh, I, O, rot, rot_dims, N):
    from mivi_v4_b200.parts.position import YarnRope
    k = K()
    x, w = rnd(N, nh, I + rot), rnd(nh * I, O, seed=1)
    pos = torch.tensor([(37 * n) % 1000 for n in range(N)])
    s = {"factor": 6.0, "original": 200, "fast": 16.0, "slow": 1.0}
    rope = YarnRope(rot_dims, 1e4, style="interleaved", **s)
    inv = rope.rotary(DEV)[0]
    assert inv.tolist() == pytest.approx(P.frequencies(1e4, rot_dims, s), rel=1e-6)
    want = P.rotate_pairs(x[..., I:], pos, {"base": 1e4, "dims": rot_dims, "scaling": s})
    order = list(range(0, rot_dims, 2)) + list(range(1, rot_dims, 2)) + list(range(rot_dims, rot))
    xp = torch.cat([x[..., :I], x[..., I:][..., order]], -1)      # the kernels pair i with i + rot_dims / 2
    y = torch.full((N, nh, O + rot), float("nan"), device=DEV)
    k.head_product(dev(xp), dev(w), y, nh, I, O, transposed=True, rot=rot, rot_dims=rot_dims, inv_freq=inv, positions=i32(pos.tolist()),
                   amplitude=rope.amplitude())
    close(y[..., :O], torch.einsum("nhi,hio->nho", x[..., :I], w.view(nh, I, O)), 1e-5, "product")
    close(y[..., O:], want[..., order], 2e-4, "tail")
    q = torch.full((N, nh, I + rot), float("nan"), dtype=BF, device=DEV)
    k.latent_query(dev(xp.reshape(N, -1)), 0, inv, i32(pos.tolist()), q, nh, I, rot, rot_dims, rope.amplitude())
    close(q, torch.cat([x[..., :I], want[..., order]], -1), 5e-3, "queries of long steps")


# ------------------------------------------------------------------------------------------ feed-forwards
def grouped(wg, wu, G=16):
    F, H = wg.shape
    return torch.stack([wg.view(F // G, G, H), wu.view(F // G, G, H)], dim=1).reshape(2 * F, H).contiguous()


@pytest.mark.parametrize("group", [0, 16])
@pytest.mark.parametrize("out_dtype", DTYPES)
def test_gelu_of_the_gate_times_up(out_dtype, group):
    k = K()
    N, F = 7, 48
    g, u = rnd(N, F, scale=3.0), rnd(N, F, seed=1)
    g[0, :6] = torch.tensor([-40.0, 40.0, 0.0, -9.0, 1e-4, -1e4])
    gu = torch.cat([g, u], 1) if not group else \
        torch.stack([g.view(N, F // group, group), u.view(N, F // group, group)], 2).reshape(N, 2 * F)
    out = torch.full((N, F), float("nan"), dtype=out_dtype, device=DEV)
    k.swiglu(dev(gu), out, group, "gelu_tanh")
    close(out, P.gelu_tanh(g) * u, 2e-6 if out_dtype == torch.float32 else 5e-3)
    with pytest.raises(k.KernelError):
        k.swiglu(dev(gu), out, group, "relu")


@pytest.mark.parametrize("M", [1, 8, 9, 33, 64, 65, 200, 1000])
@pytest.mark.parametrize("F,Kd", [(16, 8), (64, 72), (384, 96), (5120, 520), (1040, 200)])
def test_products_that_apply_gelu(M, F, Kd):
    k = K()
    x = rnd(M, Kd).to(BF).to(DEV)
    wg, wu = rnd(F, Kd, seed=1, scale=2.0 * Kd ** -0.5).to(BF).to(DEV), rnd(F, Kd, seed=2, scale=2.0 * Kd ** -0.5).to(BF).to(DEV)
    if F > 16:
        wg[:2] *= 40.0                                           # gates far out on both sides
        wg[2] = 0.0
    want = (P.gelu_tanh(x.double() @ wg.double().T) * (x.double() @ wu.double().T)).cpu()
    many = [functools.partial(k.gemm_tc, pair=False), k.gemm_tc_swap] + \
        ([functools.partial(k.gemm_tc, pair=True)] if M > 128 and 2 * F >= 128 else [])
    for fn in ([k.gemm_small_m, k.gemm_tc_swap] if M <= 64 else many):
        out = torch.full((M, F), float("nan"), dtype=BF, device=DEV)
        fn(x, grouped(wg, wu), out, swiglu=True, act="gelu_tanh")
        k.check_device_errors()
        close(out, want, 1e-2, str(fn))


@pytest.mark.parametrize("M", [1, 64, 65, 200, 1000])
@pytest.mark.parametrize("E,ff,S,Kd", [(1, 16, 0, 8), (3, 48, 16, 72), (8, 256, 128, 96), (5, 32, 0, 520), (40, 64, 64, 200)])
def test_products_with_a_weight_a_row_and_an_expert(M, E, ff, S, Kd):
    k = K()
    F = E * ff + S
    x = rnd(M, Kd).to(BF).to(DEV)
    wg, wu = rnd(F, Kd, seed=1, scale=2.0 * Kd ** -0.5).to(BF).to(DEV), rnd(F, Kd, seed=2, scale=2.0 * Kd ** -0.5).to(BF).to(DEV)
    dense = torch.rand(M, E + 2, generator=torch.Generator().manual_seed(E), dtype=F64)
    dense[:, 0:E:3] = 0.0
    wt = torch.cat([dense[:, :E].repeat_interleave(ff, 1), torch.ones(M, S, dtype=F64)], 1)
    a, b = (x.double() @ wg.double().T).cpu() * wt, (x.double() @ wu.double().T).cpu() * wt
    for pair in (False, True) if M > 128 and 2 * F >= 128 else (False,):
        out = torch.full((M, F), float("nan"), dtype=BF, device=DEV)
        k.gemm_tc(x, grouped(wg, wu), out, swiglu=True, pair=pair, weights=k.ExpertWeights(dev(dense), E, ff))
        k.check_device_errors()
        close(out, P.silu(a) * b, 1e-2, f"pair {pair}")
    with pytest.raises(k.KernelError):
        k.gemm_tc(x, grouped(wg, wu), out, swiglu=True, weights=k.ExpertWeights(dev(dense), E, ff), act="gelu_tanh")


@pytest.mark.parametrize("H,ff", [(64, 48), (40, 30), (52, 64), (128, 256)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_feed_forward_with_gelu(H, ff, dtype):
    from mivi_v4_b200.parts import PartSpec, build
    p = {"gate": rnd(ff, H, seed=1, scale=2.0 * H ** -0.5), "up": rnd(ff, H, seed=2, scale=H ** -0.5), "down": rnd(H, ff, seed=3, scale=ff ** -0.5)}
    p = {n: v.to(dtype).double() for n, v in p.items()}
    part = build("feed_forward", PartSpec("swiglu", dict(hidden=H, ff=ff, act="gelu_tanh")))
    part.load({"w1.weight": dev(p["gate"], dtype), "w3.weight": dev(p["up"], dtype), "w2.weight": dev(p["down"], dtype)})
    for N in (1, 9, 70, 300):
        h = rnd(N, H, seed=N).to(dtype).double()
        y = torch.full((N, H), float("nan"), device=DEV)
        part.forward(dev(h, dtype), y, make_step([N], [0], dtype, [[0]]), accumulate=False)
        K().check_device_errors()
        close(y, P.dense(h, p), 2e-5 if dtype == torch.float32 else 1.5e-2, f"{N} rows")


@pytest.mark.parametrize("E,top", [(6, 2), (5, 1), (3, 3), (1, 1), (40, 6), (64, 32), (130, 4)])
def test_router_without_renormalization(E, top):
    k = K()
    N = 57
    z = rnd(N, E, seed=E, scale=2.0).float().double()
    want = P.route(z, top)
    dense = torch.full((N, E), float("nan"), device=DEV)
    pick, pick_w = torch.zeros(N, top, dtype=torch.int32, device=DEV), torch.zeros(N, top, device=DEV)
    k.route(dev(z), dense, pick, pick_w, E, 1, 1, top, False, renormalize=False)
    close(dense, want, 1e-6, "dense weights")
    rows = torch.arange(N)[:, None].expand(N, top)
    close(pick_w, want[rows, pick.cpu().long()], 1e-6, "picked weights")
    k.route(dev(z), dense, pick, pick_w, E, 1, 1, top, False, renormalize=False, out_scale=2.5)
    close(dense, 2.5 * want, 1e-6, "scaled")
    k.route(dev(z), dense, pick, pick_w, E, 1, 1, top, False)
    close(dense, want / want.sum(-1, keepdim=True), 1e-6, "renormalized")


MIXTURES = [(64, dict(expert=dict(ff=32), shared=dict(ff=48), router=dict(experts=6, top=2))),
            (40, dict(expert=dict(ff=16), router=dict(experts=3, top=1))),
            (72, dict(expert=dict(ff=20), shared=dict(ff=10), router=dict(experts=5, top=5))),
            (128, dict(expert=dict(ff=64), shared=dict(ff=20), router=dict(experts=8, top=4))),
            (48, dict(expert=dict(ff=48), shared=dict(ff=48), router=dict(experts=1, top=1))),
            (51, dict(expert=dict(ff=32), shared=dict(ff=16), router=dict(experts=2, top=1)))]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,mlp", MIXTURES)
def test_mixture_whose_weights_multiply_its_inputs(H, mlp, dtype, monkeypatch):
    """Few rows, more rows than the gated products start from, and rows sorted by expert; weights small enough that
    multiplying the experts' outputs instead would show."""
    from mivi_v4_b200.parts import PartSpec, build
    from mivi_v4_b200.parts.feed_forward import RoutedExperts
    E, top, ff, sh = mlp["router"]["experts"], mlp["router"]["top"], mlp["expert"]["ff"], (mlp.get("shared") or {}).get("ff", 0)
    u = rnd(H, seed=H)
    u = u / u.norm()
    order = torch.randperm(E, generator=torch.Generator().manual_seed(H))
    p = {"router": torch.linspace(-0.6, 0.4, E, dtype=F64)[order][:, None] * u}
    for n, f in [(f"e{i}.", ff) for i in range(E)] + ([("shared.", sh)] if sh else []):
        c = len(p)
        p.update({n + "gate": rnd(f, H, seed=c, scale=2.5 * H ** -0.5), n + "up": rnd(f, H, seed=c + 1, scale=2.0 * H ** -0.5),
                  n + "down": rnd(H, f, seed=c + 2, scale=f ** -0.5)})
    p = {n: v.to(dtype).double() for n, v in p.items()}
    for lowered in (False, True):
        if lowered:
            monkeypatch.setattr(RoutedExperts, "SORTED_ROWS_AN_EXPERT", 1)
        part = build("feed_forward", PartSpec("routed_experts", dict(hidden=H, n_experts=E, ff=ff, top=top, renormalize=False,
                                                                     weight_on="input", shared_ff=sh, shared_gate=False)))
        part.load({n: dev(v, dtype) for n, v in p.items()})
        for N in (1, 8, 50, 70, 300):
            h = rnd(N, H, seed=N)
            h = h - (h @ u)[:, None] * u + torch.where(torch.arange(N) % 3 == 0, 3.0, -2.5)[:, None].double() * u    # no close calls
            h = h.to(dtype).double()
            want = P.moe(h, p, mlp)
            outputs = sum(P.route(h @ p["router"].T, top)[:, e:e + 1] * P.expert(h, p, prefix=f"e{e}.") for e in range(E)) + \
                (P.expert(h, p, prefix="shared.") if sh else 0.0)
            assert (outputs - want).abs().max() > 0.04 * want.abs().max()
            step = make_step([N], [0], dtype, [[0]])
            y = torch.full((N, H), float("nan"), device=DEV)
            part.forward(dev(h, dtype), y, step, accumulate=False)
            K().check_device_errors()
            close(y, want, 2e-5 if dtype == torch.float32 else 1.5e-2, f"{N} rows, sorted {lowered}")
            part.forward(dev(h, dtype), y, step)                       # and added to what is there
            close(y, 2.0 * want, 2e-5 if dtype == torch.float32 else 1.5e-2, f"{N} rows twice, sorted {lowered}")
