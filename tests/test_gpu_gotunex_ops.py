"""GPU: the kernels of the Gotunex design, each alone, against the plain implementation in float64."""
from __future__ import annotations

import math

import pytest
import torch

from oracle import gotunex_oracle as go
from spikeinfer_b200.attention import PrefillPlan
from spikeinfer_b200.engine.kv_state_cache import PagedLatentPool
from spikeinfer_b200.kernels import delta as kd
from spikeinfer_b200.kernels import dense as kn
from spikeinfer_b200.kernels import experts as ke
from spikeinfer_b200.kernels import latent as kl
from spikeinfer_b200.rotary import RotaryConfig

pytestmark = pytest.mark.gpu
F32, BF = torch.float32, torch.bfloat16
DTYPES = [F32, BF]
TOL = {F32: 2e-6, BF: 1.2e-2}


def gen(seed):
    return torch.Generator().manual_seed(seed)


def rel(got, want) -> float:
    want = want.double()
    return float((got.double().cpu() - want).pow(2).mean().sqrt() / want.pow(2).mean().sqrt().clamp(min=1e-30))


@pytest.fixture
def status(dev):
    s = torch.zeros(1, dtype=torch.int32, device=dev)
    yield s
    assert int(s.item()) == 0


# ---- boundary and activation -----------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,width,top", [(1, 45, 1), (37, 88, 3), (5, 1030, 2), (64, 3584, 4), (3, 9000, 2)])
def test_boundary(dev, status, n, width, top, dtype):
    g = gen(n + width)
    rnd = lambda *s: torch.randn(*s, generator=g)
    x, delta, w1, w2, eps, scale = rnd(n, width), rnd(n, width), rnd(width), rnd(width), 1e-3, 0.37
    rows = 8 * (-(-n * top // 8)) + 8
    slots = torch.randperm(rows, generator=g)[: n * top].view(n, top).to(torch.int32)
    slots[0, 0] = -1
    pairs = rnd(rows, width)
    pairs[[r for r in range(rows) if r not in slots.flatten().tolist()]] = float("nan")
    y = x.double() + delta.double()
    for t in range(n):
        for s in slots[t].tolist():
            if s >= 0:
                y[t] += scale * pairs[s].double()
    d = lambda t: t.to(dev)
    xo, o1 = d(x), torch.empty(n, width, dtype=dtype, device=dev)
    tiled = dtype == BF
    o2 = torch.full((-(-width // 64), rows, 64) if tiled else (rows, width), float("nan"), dtype=dtype, device=dev)
    kn.rms_residual(eps=eps, x=xo, delta=d(delta), x_out=xo, pairs=d(pairs), pair_slots=d(slots), pair_scale=scale, w1=d(w1), out1=o1, w2=d(w2),
                    out2=o2, out2_slots=d(slots), out2_tiled=tiled, status=status)
    assert rel(xo, y) < 1e-6
    assert rel(o1, go.rms(y, eps) * w1) < (1e-6 if dtype == F32 else 4e-3)
    if tiled:
        k = -(-width // 64) * 64
        o2 = ke.plain_rows(o2, k)
        used = [s for s in slots.flatten().tolist() if s >= 0]
        assert (o2[used, width:] == 0).all()
        o2 = o2[:, :width]
    want = go.rms(y, eps) * w2
    for t in range(n):
        for s in slots[t].tolist():
            if s >= 0:
                assert rel(o2[s], want[t]) < (2e-6 if dtype == F32 else 6e-3)
    # the embedding row, and a dense second output
    table, ids = rnd(50, width).to(dtype), torch.randint(0, 50, (n,), generator=g)
    o2 = torch.empty_like(o1)
    kn.rms_residual(eps=eps, ids=d(ids), embed=d(table), embed_scale=1.7, x_out=xo, w1=d(w1), out1=o1, w2=d(w2), out2=o2, status=status)
    y = table[ids].double() * 1.7
    assert rel(xo, y) < 1e-6 and rel(o2, go.rms(y, eps) * w2) < (1e-6 if dtype == F32 else 4e-3)


@pytest.mark.parametrize("dtype", DTYPES)
def test_gelu(dev, dtype):
    z = torch.linspace(-9, 9, 3 * 41).view(3, 41).to(dtype)
    out = torch.zeros(3, 60, dtype=dtype, device=dev)
    kn.gelu_tanh(z.to(dev), out[:, 7:48])
    assert (out[:, :7] == 0).all() and (out[:, 48:] == 0).all()
    err = (out[:, 7:48].double().cpu() - go.gelu_tanh(z.double())).abs().max()
    assert err < (2e-6 if dtype == F32 else 4e-2)


# ---- experts ---------------------------------------------------------------------------------------------------------
def expert_case(dev, dtype, n, width, experts, top, ff, seed, ids=None, vocab=61):
    g = gen(seed)
    mat = lambda o, i: (torch.randn(o, i, generator=g) / math.sqrt(i)).to(BF)
    w = {}
    for e in range(experts):
        w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"] = mat(ff, width), mat(ff, width), mat(width, ff)
    w["table"] = torch.stack([torch.randperm(experts, generator=g)[:top] for _ in range(vocab)]).to(torch.int32)
    part = lambda name: [w[f"e{e}.{name}"].to(dev, dtype) for e in range(experts)]
    weights = ke.ExpertWeights(part("gate"), part("up"), part("down"), w["table"].to(dev))
    ids = torch.randint(0, vocab, (n,), generator=g) if ids is None else ids
    return w, weights, ids, torch.randn(n, width, generator=g).to(dtype), dict(router=dict(experts=experts, top=top))


def run_experts(dev, status, weights, ids, x, active=None):
    vocab = weights.table.shape[0]
    route = ke.ExpertRouter([weights], vocab)(ids.to(dev), active, status)[0]
    n, width = x.shape
    ones = torch.ones(width, device=dev)
    xs = weights.sorted_matrix(n, width)
    xs.fill_(float("nan"))
    # a norm of weight root-mean-square hands the rows on as they are: use rows of unit mean square
    kn.rms_residual(eps=0.0, x=x.float().to(dev), w1=ones, out1=torch.empty(n, width, dtype=weights.dtype, device=dev), w2=ones, out2=xs,
                    out2_slots=route.slots, out2_tiled=weights.tiled, status=status)
    return route, ke.experts_forward(xs, weights, route, status)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,width,experts,top,ff", [(1, 45, 2, 2, 9), (5, 88, 7, 3, 40), (130, 72, 5, 1, 200), (300, 130, 3, 2, 136),
                                                    (700, 64, 4, 2, 64), (33, 320, 64, 4, 257), (250, 72, 4, 1, 96)])
def test_experts(dev, status, n, width, experts, top, ff, dtype):
    w, weights, ids, x, cfg = expert_case(dev, dtype, n, width, experts, top, ff, n + ff)
    x = go.rms(x.double(), 0.0)
    route, out = run_experts(dev, status, weights, ids, x)
    slots = route.slots.cpu()
    assert sorted(slots.flatten().tolist()) == sorted({*slots.flatten().tolist()})      # a row per pair
    assert int((route.segs[:, 0] % 8).sum()) == 0 and int(route.segs[:, 1].sum()) == n * top
    got = out.cpu().double()[slots.long()].mean(1)
    want = go.table_experts(x, ids.tolist(), go.as_float(w), "", cfg)
    assert rel(got, want) < (3e-6 if dtype == F32 else 8e-3)


@pytest.mark.parametrize("dtype", DTYPES)
def test_every_token_at_the_same_experts_and_rows_that_sit_out(dev, status, dtype):
    n = 150
    ids = torch.full((n,), 7)
    w, weights, ids, x, cfg = expert_case(dev, dtype, n, 96, 9, 2, 48, 3, ids=ids)
    x = go.rms(x.double(), 0.0)
    active = torch.ones(n, dtype=torch.int32, device=dev)
    active[[0, 17, 149]] = 0
    route, out = run_experts(dev, status, weights, ids, x, active)
    slots = route.slots.cpu().long()
    assert (slots[[0, 17, 149]] == -1).all() and int(route.segs[:, 1].sum()) == (n - 3) * 2 and int((route.segs[:, 1] > 0).sum()) == 2
    live = [t for t in range(n) if t not in (0, 17, 149)]
    want = go.table_experts(x, ids.tolist(), go.as_float(w), "", cfg)[live]
    assert rel(out.cpu().double()[slots[live]].mean(1), want) < (3e-6 if dtype == F32 else 8e-3)


def test_routing_of_several_layers_at_once(dev, status):
    layers = [expert_case(dev, F32, 4, 8, e, t, 8, e)[1] for e, t in ((40, 3), (5, 1), (33, 7))]
    ids = torch.randint(0, 61, (2000,), generator=gen(1))
    for w, r in zip(layers, ke.ExpertRouter(layers, 61)(ids.to(dev), None, status)):
        segs, slots = r.segs.cpu(), r.slots.cpu()
        want = w.table.cpu()[ids]
        ends = segs[:, 0] + segs[:, 1]
        assert (segs[1:, 0] >= ends[:-1]).all() and int(ends.max()) <= w.rows(2000)
        owner = torch.searchsorted(segs[:, 0].contiguous(), slots.flatten().to(torch.int32), right=True) - 1
        # empty segments share their start with the next one: compare by range
        ok = (slots >= segs[want.long(), 0]) & (slots < ends[want.long()])
        assert ok.all() and owner.numel() == ok.numel() and slots.unique().numel() == slots.numel()


# ---- latent attention ------------------------------------------------------------------------------------------------
def filled_pool(dev, dtype, seqs, rank, rot_dim, block_size, seed, blocks=None):
    """Cache rows of several sequences in shuffled pages; every other row, the ones after a sequence's end included, is NaN."""
    per = [-(-c.shape[0] // block_size) for c in seqs]
    nb = sum(per) + 3 if blocks is None else blocks
    pool = PagedLatentPool(nb, block_size, rank, rot_dim, dtype, dev)
    order = torch.randperm(nb - 1, generator=gen(seed)).tolist()
    tables = torch.full((len(seqs), max(per) + 1), nb - 1, dtype=torch.int32)
    plain = torch.full((nb * block_size, pool.pad), float("nan"))
    plain[:, rank: pool.rank_pad] = 0
    plain[:, pool.rank_pad + rot_dim:] = 0
    at = 0
    for i, c in enumerate(seqs):
        for b in range(per[i]):
            tables[i, b] = order[at]
            part = c[b * block_size: (b + 1) * block_size]
            lo = order[at] * block_size
            plain[lo: lo + part.shape[0], :rank] = part[:, :rank]
            plain[lo: lo + part.shape[0], pool.rank_pad: pool.rank_pad + rot_dim] = part[:, rank:]
            at += 1
    x = plain.view(nb, 1, block_size, pool.pad)
    if pool.tiled:
        r = torch.arange(8)
        x = x.view(nb, block_size // 8, 8, pool.pad // 64, 8, 8).transpose(2, 3)
        x = x.gather(4, (r[None, :] ^ r[:, None]).view(1, 1, 1, 8, 8, 1).expand(x.shape)).reshape(nb, 1, block_size, pool.pad)
    pool.data.copy_(x.to(dtype))
    return pool, tables.to(dev)


def attention_reference(q, c, kr, w_uk, w_uv, sink, gate, positions, rot, scale, heads, dim, vdim):
    """Queries ``[n, heads, dim + rot]`` at ``positions`` over one sequence's cache."""
    out = torch.zeros(q.shape[0], heads, vdim, dtype=torch.float64)
    for t, p in enumerate(positions):
        for h in range(heads):
            keys = c[: p + 1] @ w_uk[h * dim:(h + 1) * dim].t()
            qr = go.rotate(q[t, h, dim:], p, rot)
            s = (keys @ q[t, h, :dim] + kr[: p + 1] @ qr) * scale
            out[t, h] = go.sink_softmax(s, sink[h]) @ (c[: p + 1] @ w_uv[h * vdim:(h + 1) * vdim].t())
    return out.flatten(1) * torch.sigmoid(gate)


SIZES = [(3, 24, 16, 20, 56), (1, 7, 6, 5, 13), (17, 64, 32, 64, 256), (6, 128, 64, 128, 512), (40, 48, 64, 72, 128), (2, 140, 96, 150, 600),
         (5, 30, 20, 33, 330)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,rot_dim,vdim,rank", SIZES)
def test_prepare_and_query(dev, status, heads, dim, rot_dim, vdim, rank, dtype):
    g = gen(rank)
    n, q_rank, eps = 21, 44, 1e-4
    lo = -(-q_rank // 8) * 8
    z = torch.randn(n, lo + rank + rot_dim + 3, generator=g).to(dtype)
    wq, wkv = torch.rand(q_rank, generator=g) + 0.5, torch.rand(rank, generator=g) + 0.5
    rot = dict(dims=rot_dim, base=3000.0)
    table = RotaryConfig(rot_dim, 3000.0).table(200, dev)
    pos = torch.randint(0, 200, (n,), generator=g)
    slots = torch.randperm(5 * 16, generator=g)[:n]
    pool = PagedLatentPool(5, 16, rank, rot_dim, dtype, dev)
    zd = z.to(dev)
    cq = kl.latent_prepare(zd[:, :q_rank], wq.to(dev), eps=eps, kv=zd[:, lo: lo + rank + rot_dim], w_kv=wkv.to(dev), pool=pool, rot_table=table,
                           positions=pos.to(dev), slot_mapping=slots.to(dev), status=status)
    zz = z.double()
    tol = 2e-6 if dtype == F32 else 4e-3
    assert rel(cq, go.rms(zz[:, :q_rank], eps) * wq) < tol
    rows = pool.rows().cpu()[slots]
    assert rel(rows[:, :rank], go.rms(zz[:, lo: lo + rank], eps) * wkv) < tol
    assert rel(rows[:, rank:], torch.stack([go.rotate(zz[t, lo + rank: lo + rank + rot_dim], int(pos[t]), rot) for t in range(n)])) < tol
    q = torch.randn(n, heads * (dim + rot_dim), generator=g).to(dtype)
    w_uk = (torch.randn(heads * dim, rank, generator=g) / math.sqrt(dim)).to(dtype)
    out = kl.latent_query(q.to(dev), w_uk.to(dev), pool, table, pos.to(dev), heads=heads, dim=dim, status=status).cpu()
    qq = q.double().view(n, heads, -1)
    want = torch.einsum("nhd,hdr->nhr", qq[..., :dim], w_uk.double().view(heads, dim, rank))
    assert rel(out[..., :rank], want) < tol
    assert rel(out[..., pool.rank_pad: pool.rank_pad + rot_dim], torch.stack([go.rotate(qq[t, :, dim:], int(pos[t]), rot) for t in range(n)])) < tol
    assert (out[..., rank: pool.rank_pad] == 0).all() and (out[..., pool.rank_pad + rot_dim:] == 0).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("block_size", [16, 4, 64])
@pytest.mark.parametrize("heads,dim,rot_dim,vdim,rank", SIZES)
def test_attention_decode_and_prefill(dev, status, heads, dim, rot_dim, vdim, rank, block_size, dtype):
    g = gen(heads + rank)
    rnd = lambda *s: torch.randn(*s, generator=g)
    lens = [1, 70, 16, 131, 64]
    rot, scale = dict(dims=rot_dim, base=800.0), 0.4 / math.sqrt(dim + rot_dim)
    table = RotaryConfig(rot_dim, 800.0).table(256, dev)
    seqs = [rnd(n, rank + rot_dim).to(dtype).float() for n in lens]
    pool, tables = filled_pool(dev, dtype, seqs, rank, rot_dim, block_size, 5)
    w_uk, w_uv = ((rnd(heads * d, rank) / math.sqrt(rank)).to(dtype) for d in (dim, vdim))
    sink = rnd(heads) * 2
    sink[0] = 6.0
    f = lambda t: t.double()
    args = dict(vdim=vdim, scale=scale, status=status)
    dd = lambda t: t.to(dev)

    def reference(i, q, gate, positions):
        c = f(seqs[i])
        return attention_reference(f(q).view(len(positions), heads, -1), c[:, :rank], c[:, rank:], f(w_uk), f(w_uv), f(sink), f(gate), positions, rot, scale,
                                   heads, dim, vdim)
    # decode: one query per row at its last position, one row inactive
    n = len(lens)
    q, gate = (rnd(n, heads * (dim + rot_dim)) * 3).to(dtype), rnd(n, heads * vdim).to(dtype)
    active = torch.ones(n, dtype=torch.int32)
    active[2] = 2
    out = torch.full((n, heads * vdim), float("nan"), dtype=dtype, device=dev)
    pos = torch.tensor(lens) - 1
    ql = kl.latent_query(dd(q), dd(w_uk), pool, table, dd(pos), heads=heads, dim=dim, status=status)
    kl.latent_attention(ql, pool, tables, dd(sink), dd(w_uv), dd(gate), out, seq_lens=dd(torch.tensor(lens, dtype=torch.int32)), active=dd(active), **args)
    out = out.cpu()
    assert (out[2] == 0).all()
    for i in (0, 1, 3, 4):
        assert rel(out[i], reference(i, q[i], gate[i], [lens[i] - 1])[0]) < TOL[dtype] * (1 if dtype == F32 else 2), i
    # prefill: portions at the end of every sequence, the first positions included
    tokens = [(0, 0), *((1, p) for p in range(60, 70)), *((3, p) for p in range(0, 3)), *((3, p) for p in range(62, 67)), (3, 127), (3, 128), (3, 130)]
    m = len(tokens)
    q, gate = (rnd(m, heads * (dim + rot_dim)) * 3).to(dtype), rnd(m, heads * vdim).to(dtype)
    rows, pos = torch.tensor([r for r, _ in tokens], dtype=torch.int32), torch.tensor([p for _, p in tokens])
    out = torch.empty(m, heads * vdim + 8, dtype=dtype, device=dev)[:, : heads * vdim]
    ql = kl.latent_query(dd(q), dd(w_uk), pool, table, dd(pos), heads=heads, dim=dim, status=status)
    kl.latent_attention(ql, pool, tables, dd(sink), dd(w_uv), dd(gate), out, token_rows=dd(rows), positions=dd(pos), most_keys=131, **args)
    for t, (i, p) in enumerate(tokens):
        assert rel(out[t], reference(i, q[t], gate[t], [p])[0]) < TOL[dtype] * (1 if dtype == F32 else 2), (i, p)


@pytest.mark.parametrize("block_size", [16, 64])
@pytest.mark.parametrize("heads,dim,rot_dim,vdim,rank", [s for s in SIZES if s[1] <= 128 and s[2] <= 64])
def test_spelled_out_prefill(dev, status, heads, dim, rot_dim, vdim, rank, block_size):
    """Portions of several sequences, some behind a cached context: the form with keys and values spelled out against the plain
    implementation (a few positions of each) and against the other form (all)."""
    g = gen(heads + dim)
    rnd = lambda *s: torch.randn(*s, generator=g)
    ctx, lens, dtype = [0, 37, 200, 0, 128], [70, 5, 300, 1, 129], BF
    rot, scale = dict(dims=rot_dim, base=800.0), 0.4 / math.sqrt(dim + rot_dim)
    table = RotaryConfig(rot_dim, 800.0).table(512, dev)
    seqs = [(rnd(c + n, rank + rot_dim)).to(dtype).float() for c, n in zip(ctx, lens)]
    seqs[2][450] *= 6                                    # late scores above everything before: the reference moves
    seqs[2][451:460, :] *= 3
    pool, tables = filled_pool(dev, dtype, seqs, rank, rot_dim, block_size, 5)
    w_uk, w_uv = ((rnd(heads * d, rank) / math.sqrt(rank)).to(dtype) for d in (dim, vdim))
    sink = rnd(heads) * 2
    sink[0] = 6.0
    n = sum(lens)
    starts = [sum(lens[:i]) for i in range(5)]
    q, gate = (rnd(n, heads * (dim + rot_dim)) * 3).to(dtype), rnd(n, heads * vdim).to(dtype)
    pos = torch.cat([torch.arange(c, c + m) for c, m in zip(ctx, lens)]).to(dev)
    rows = torch.cat([torch.full((m,), i, dtype=torch.int32) for i, m in enumerate(lens)]).to(dev)
    plan = PrefillPlan(starts, lens, ctx, list(range(5)), dev)
    dd = lambda t: t.to(dev)
    w_kv = kl.spelled_out_weights(dd(w_uk), dd(w_uv), heads)
    outs = []
    for form in (True, False):
        out = torch.full((n, heads * vdim + 8), float("nan"), dtype=dtype, device=dev)[:, : heads * vdim]
        kl.latent_prefill(dd(q), pool, tables, dd(w_uk), dd(w_uv), w_kv, dd(sink), dd(gate), out, rot_table=table, positions=pos, token_rows=rows, plan=plan,
                          heads=heads, dim=dim, vdim=vdim, scale=scale, spelled_out=form, status=status)
        outs.append(out.cpu())
    assert rel(outs[0], outs[1]) < 3e-2
    f = lambda t: t.double()
    for i, picks in enumerate([(0, 1, 15, 16, 63, 64, 69), (0, 4), (0, 55, 56, 183, 184, 249, 250, 251, 299), (0,), (0, 1, 127, 128)]):
        t = [starts[i] + p for p in picks]
        c = f(seqs[i])
        want = attention_reference(f(q[t]).view(len(t), heads, -1), c[:, :rank], c[:, rank:], f(w_uk), f(w_uv), f(sink), f(gate[t]),
                                   [ctx[i] + p for p in picks], rot, scale, heads, dim, vdim)
        for k in range(len(t)):
            assert rel(outs[0][t[k]], want[k]) < 2.4e-2, (i, picks[k])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,rank", [(2, 56), (20, 256), (4, 512)])
def test_one_key_stands_out(dev, status, heads, rank, dtype):
    """A single loud key among a thousand, at page, tile and range borders: the query at its position and later sees it, the one just
    before does not."""
    dim, rot_dim, vdim, n = 16, 16, 16, 1400
    table = RotaryConfig(rot_dim, 1e4).table(n, dev)
    g = gen(9)
    w_uk = torch.zeros(heads * dim, rank)
    w_uv = torch.zeros(heads * vdim, rank)
    for h in range(heads):
        w_uk[h * dim: (h + 1) * dim, :dim] = torch.eye(dim)
        w_uv[h * vdim: (h + 1) * vdim, rank - vdim:] = torch.eye(vdim)
    for j in (0, 1, 15, 16, 63, 64, 127, 128, 255, 256, 511, 512, 703, 704, 1023, 1279, 1280, 1398):
        c = torch.zeros(n, rank + rot_dim)
        c[:, rank - vdim: rank] = torch.randn(n, vdim, generator=g) * 0.01
        c[j, :dim] = 4.0
        c[j, rank - vdim: rank] = torch.arange(1, vdim + 1).float()
        pool, tables = filled_pool(dev, dtype, [c], rank, rot_dim, 16, 3)
        q = torch.zeros(3, heads, dim + rot_dim)
        q[..., :dim] = 1.0
        where = [max(j - 1, 0), j, n - 1]
        pos = torch.tensor(where)
        dd = lambda t: t.to(dev)
        ql = kl.latent_query(dd(q.flatten(1).to(dtype)), dd(w_uk.to(dtype)), pool, table, dd(pos), heads=heads, dim=dim, status=status)
        gate = torch.full((3, heads * vdim), 30.0, dtype=dtype, device=dev)
        loud = torch.arange(1, vdim + 1).float().repeat(heads)
        sink = torch.full((heads,), -5.0, device=dev)
        out = torch.empty(3, heads * vdim, dtype=dtype, device=dev)
        kl.latent_attention(ql, pool, tables, sink, dd(w_uv.to(dtype)), gate, out, vdim=vdim, scale=0.5, token_rows=torch.zeros(3, dtype=torch.int32, device=dev),
                            positions=dd(pos), most_keys=n, status=status)
        single = torch.empty(1, heads * vdim, dtype=dtype, device=dev)
        kl.latent_attention(ql[2:], pool, tables, sink, dd(w_uv.to(dtype)), gate[:1], single, vdim=vdim, scale=0.5,
                            seq_lens=torch.tensor([n], dtype=torch.int32, device=dev), status=status)
        for row in (out[1], out[2], single[0]):
            assert (row.float().cpu() - loud).abs().max() < 0.1, j
        if j > 0:
            assert out[0].abs().max() < 0.1, j
        if dtype == BF:  # a whole portion, keys and values spelled out
            m = 320
            lo = min(max(j - 100, 0), n - m)
            plan = PrefillPlan([0], [m], [lo], [0], dev)
            qs = dd(q[:1].flatten(1).to(dtype)).expand(m, -1).contiguous()
            full = torch.empty(m, heads * vdim, dtype=dtype, device=dev)
            kl.latent_prefill(qs, pool, tables, dd(w_uk.to(dtype)), dd(w_uv.to(dtype)), kl.spelled_out_weights(dd(w_uk.to(dtype)), dd(w_uv.to(dtype)), heads),
                              sink, gate[:1].expand(m, -1).contiguous(), full, rot_table=table, positions=torch.arange(lo, lo + m, device=dev),
                              token_rows=torch.zeros(m, dtype=torch.int32, device=dev), plan=plan, heads=heads, dim=dim, vdim=vdim, scale=0.5,
                              spelled_out=True, status=status)
            assert (full[j - lo:].float().cpu() - loud).abs().max() < 0.1, j
            if j > lo:
                assert full[: j - lo].abs().max() < 0.1, j


def test_a_sink_takes_its_share(dev, status):
    """Equal scores s over n keys: the output is n e^s / (n e^s + e^sink) of the mean, whatever the scale of the scores."""
    rank, rot_dim, heads, dim, vdim, n = 64, 16, 4, 8, 8, 200
    table = RotaryConfig(rot_dim, 1e4).table(n, dev)
    for dtype in DTYPES:
        c = torch.zeros(n, rank + rot_dim)
        c[:, 0] = 1.0
        c[:, 8] = 1.0
        pool, tables = filled_pool(dev, dtype, [c], rank, rot_dim, 16, 3)
        w_uk, w_uv = torch.zeros(heads * dim, rank), torch.zeros(heads * vdim, rank)
        w_uk[::dim, 0] = 1.0
        w_uv[:, 8] = 1.0
        q = torch.zeros(1, heads, dim + rot_dim)
        q[0, :, 0] = torch.tensor([-200.0, 0.0, 8.0, 400.0])
        sink = torch.tensor([-100.0 + math.log(n), 5.0, 6.0, 0.0])
        ql = kl.latent_query(q.flatten(1).to(dtype).to(dev), w_uk.to(dtype).to(dev), pool, table, torch.tensor([n - 1], device=dev), heads=heads, dim=dim)
        gate = torch.full((1, heads * vdim), 30.0, dtype=dtype, device=dev)
        out = torch.empty(1, heads * vdim, dtype=dtype, device=dev)
        kl.latent_attention(ql, pool, tables, sink.to(dev), w_uv.to(dtype).to(dev), gate, out, vdim=vdim, scale=0.5,
                            seq_lens=torch.tensor([n], dtype=torch.int32, device=dev), status=status)
        s = torch.tensor([-100.0, 0.0, 4.0, 200.0]).double()
        want = torch.sigmoid(s + math.log(n) - sink.double()).repeat_interleave(vdim)
        assert (out[0].double().cpu() - want).abs().max() < (1e-5 if dtype == F32 else 4e-3), dtype


# ---- gated delta rule ------------------------------------------------------------------------------------------------
class DeltaCase:
    def __init__(self, dev, dtype, n, heads, kv_heads, dim, vdim, taps, seed, decay=(-5.0, 0.5), rows=3):
        g = gen(seed)
        rnd = lambda *s: torch.randn(*s, generator=g)
        self.sizes, self.dev, self.dtype, self.eps = (heads, kv_heads, dim, vdim, taps), dev, dtype, 1e-4
        qk, v = kv_heads * dim, heads * vdim
        self.z = rnd(n, 2 * qk + v + heads).to(dtype)
        self.y = (rnd(n, heads * dim + v)).to(dtype)
        self.conv = [rnd(r, taps) * 0.7 for r in (qk, qk, v)]
        self.a_log, self.norm = torch.rand(heads, generator=g) * 3 - 2, torch.rand(vdim, generator=g) + 0.5
        self.dt_bias = decay[0] + (decay[1] - decay[0]) * torch.rand(heads * dim, generator=g)
        self.widths = [qk, qk, v, heads]
        nan = float("nan")
        self.state = torch.full((rows, heads, dim, vdim), nan, device=dev)
        self.conv_state = torch.full((rows, taps, 2 * qk + v), nan, device=dev)

    def want(self):
        heads, kv_heads, dim, vdim, _ = self.sizes
        n = self.z.shape[0]
        q, k, v, b = self.z.double().split(self.widths, dim=1)
        act = lambda x, w: go.silu(go.causal_conv(x, w.double()))
        q = go.unit(act(q, self.conv[0]).view(n, kv_heads, dim)) * dim ** -0.5
        k = go.unit(act(k, self.conv[1]).view(n, kv_heads, dim))
        v = act(v, self.conv[2]).view(n, heads, vdim)
        raw, gate = self.y.double().split([heads * dim, heads * vdim], dim=1)
        log_decay = (-torch.exp(self.a_log.double())[None, :, None] * go.softplus(raw + self.dt_bias.double()).view(n, heads, dim))
        out, states = torch.zeros(n, heads, vdim, dtype=torch.float64), []
        for h in range(heads):
            g = h // (heads // kv_heads)
            o, S = go.delta_rule(q[:, g], k[:, g], v[:, h], torch.sigmoid(b[:, h]), log_decay[:, h])
            out[:, h] = go.rms(o, self.eps) * self.norm.double()
            states.append(S)
        return out.flatten(1) * torch.sigmoid(gate), torch.stack(states)

    def run(self, lo, hi, row, status, decode=False, rows=3):
        """Tokens lo .. hi - 1: a prefill portion in `row`, or decode steps with the other rows sitting out."""
        heads, kv_heads, dim, vdim, _ = self.sizes
        dd = lambda t: t.to(self.dev)
        common = dict(conv=[dd(c) for c in self.conv], a_log=dd(self.a_log), dt_bias=dd(self.dt_bias), norm=dd(self.norm), state=self.state,
                      conv_state=self.conv_state, kv_heads=kv_heads, eps=self.eps, status=status)
        split = lambda z, y: (*dd(z).split(self.widths, dim=1), *dd(y).split([heads * dim, heads * vdim], dim=1))
        if not decode:
            out = torch.empty(hi - lo, heads * vdim, dtype=self.dtype, device=self.dev)
            plan = PrefillPlan([0], [hi - lo], [lo], [row], self.dev)
            return kd.delta_rule(*split(self.z[lo:hi], self.y[lo:hi]), out=out, plan=plan, **common).cpu()
        outs = []
        active = torch.full((rows,), 2, dtype=torch.int32)
        active[row] = 1
        for t in range(lo, hi):
            z, y = (x[t:t + 1].expand(rows, -1).contiguous() for x in (self.z, self.y))
            out = torch.empty(rows, heads * vdim, dtype=self.dtype, device=self.dev)
            pos = torch.full((rows,), t, dtype=torch.int64)
            kd.delta_rule(*split(z, y), out=out, positions=dd(pos), active=dd(active), **common)
            assert (out.cpu()[[r for r in range(rows) if r != row]] == 0).all()
            outs.append(out[row].cpu())
        return torch.stack(outs)


DELTA_SIZES = [(4, 2, 24, 40, 4), (3, 1, 10, 7, 1), (2, 2, 13, 21, 6), (4, 2, 64, 64, 4), (2, 1, 128, 128, 4), (2, 1, 160, 144, 2), (3, 3, 32, 130, 3),
               (2, 2, 100, 36, 4), (1, 1, 300, 20, 3)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,taps", DELTA_SIZES)
def test_delta_prefill_portions_and_decode(dev, status, heads, kv_heads, dim, vdim, taps, dtype):
    n = 190
    case = DeltaCase(dev, dtype, n, heads, kv_heads, dim, vdim, taps, dim + vdim)
    want, state = case.want()
    tol = 4e-6 if dtype == F32 else 8e-3
    got = case.run(0, n, 1, status)
    assert rel(got, want) < tol and rel(case.state[1], state) < tol
    at = 0
    for size in (2, 1, 3, 64, 2, 15, 66, 2):          # the same slot again, in portions: what it holds does not show
        assert rel(case.run(at, at + size, 1, status), want[at:at + size]) < tol, at
        at += size
    assert rel(case.run(at, at + 9, 1, status, decode=True), want[at:at + 9]) < tol
    at += 9
    assert rel(case.run(at, n, 1, status), want[at:]) < tol          # a portion after decode steps
    assert rel(case.state[1], state) < tol
    assert torch.isnan(case.state[[0, 2]]).all() and torch.isnan(case.conv_state[[0, 2]]).all()
    got = case.run(0, 40, 0, status, decode=True)                      # from the first token on, in a used slot
    assert rel(got, want[:40]) < tol


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decay", [(20.0, 60.0), (-30.0, -20.0), (-8.0, 12.0), (1.0, 3.0), (3.0, 5.0)])
@pytest.mark.parametrize("dim,vdim", [(64, 64), (128, 128), (40, 24)])
def test_delta_with_extreme_decays(dev, status, decay, dim, vdim, dtype):
    """Decays that wipe the state in one step, that keep it for good, both side by side, and strong ones a chunk just can or cannot
    divide by."""
    n = 150
    case = DeltaCase(dev, dtype, n, 2, 1, dim, vdim, 4, 11, decay=decay)
    want, state = case.want()
    tol = 1e-5 if dtype == F32 else 1e-2
    assert rel(case.run(0, 70, 2, status), want[:70]) < tol
    assert rel(case.run(70, 75, 2, status, decode=True), want[70:75]) < tol
    assert rel(case.run(75, n, 2, status), want[75:]) < tol
    if decay[0] < 0:
        assert rel(case.state[2], state) < tol


@pytest.mark.parametrize("dtype", DTYPES)
def test_delta_portions_of_several_requests_at_once(dev, status, dtype):
    heads, kv_heads, dim, vdim, taps = 4, 2, 64, 64, 4
    cases = [DeltaCase(dev, dtype, n, heads, kv_heads, dim, vdim, taps, 40 + n) for n in (5, 150, 64, 1)]
    one = cases[0]
    for c in cases[1:]:
        c.conv, c.a_log, c.dt_bias, c.norm = one.conv, one.a_log, one.dt_bias, one.norm
    state, conv_state = torch.full((6, heads, dim, vdim), float("nan"), device=dev), torch.full((6, taps, 2 * kv_heads * dim + heads * vdim), float("nan"), device=dev)
    rows, lens = [4, 0, 5, 2], [c.z.shape[0] for c in cases]
    starts = [sum(lens[:i]) for i in range(4)]
    z, y = torch.cat([c.z for c in cases]).to(dev), torch.cat([c.y for c in cases]).to(dev)
    out = torch.empty(sum(lens), heads * vdim, dtype=dtype, device=dev)
    kd.delta_rule(*z.split(one.widths, dim=1), *y.split([heads * dim, heads * vdim], dim=1), conv=[c.to(dev) for c in one.conv], a_log=one.a_log.to(dev),
                  dt_bias=one.dt_bias.to(dev), norm=one.norm.to(dev), state=state, conv_state=conv_state, out=out, kv_heads=kv_heads, eps=one.eps,
                  plan=PrefillPlan(starts, lens, [0] * 4, rows, dev), status=status)
    tol = 4e-6 if dtype == F32 else 8e-3
    for c, s, n, r in zip(cases, starts, lens, rows):
        want, S = c.want()
        assert rel(out[s:s + n], want) < tol and rel(state[r], S) < tol
    assert torch.isnan(state[[1, 3]]).all()
