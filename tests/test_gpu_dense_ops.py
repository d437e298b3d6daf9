"""GPU: every mechanism of the dense decoder kernels alone, against the plain implementation in float64 on the same inputs.

Inputs are made so that a fault shows: single keys that outweigh all others at page, tile and range borders, future keys and
stale page rows that would, states and slots full of NaN that must not be read."""
from __future__ import annotations

import pytest
import torch

from oracle import manirax_oracle as mo
from spikeinfer_b200 import _lib
from spikeinfer_b200.attention import PrefillPlan
from spikeinfer_b200.engine.batch_state import DecodeBatchState
from spikeinfer_b200.engine.kv_state_cache import PagedKVPool
from spikeinfer_b200.kernels import dense

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]
TOL = {torch.float32: 3e-6, torch.bfloat16: 6e-3}


def rel(got, want) -> float:
    got, want = got.double().cpu(), want.double().cpu()
    assert torch.isfinite(got).all()
    return float((got - want).abs().max() / want.abs().max().clamp(min=1e-9))


def gen(seed):
    return torch.Generator().manual_seed(seed)


# ---- residual boundary -------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [24, 37, 130, 1152, 5000])
def test_residual_norm_portions(dev, dtype, width):
    """Three portions, one continuing a sequence, one of a single token; shift, commit and both norms."""
    g = gen(width)
    lens, contexts, rows = [5, 1, 700 if width < 200 else 9], [3, 0, 0], [2, 0, 4]
    n = sum(lens)
    x, delta = torch.randn(n, width, generator=g), torch.randn(n, width, generator=g)
    w, w2 = 1 + 0.3 * torch.randn(width, generator=g), 1 + 0.3 * torch.randn(width, generator=g)
    mix = torch.rand(width, generator=g)
    prev = torch.randn(6, width, generator=g)
    prev[4] = float("nan")  # a new sequence's slot may hold anything
    prev[0] = float("nan")
    eps, alpha = 1e-3, 2.5
    pos = torch.cat([torch.arange(c, c + m) for c, m in zip(contexts, lens)]).to(dev)
    trow = torch.cat([torch.full((m,), r, dtype=torch.int32) for r, m in zip(rows, lens)]).to(dev)
    edge = torch.zeros(n, dtype=torch.int32)
    at = 0
    for m in lens:
        edge[at] |= 1
        edge[at + m - 1] |= 2
        at += m
    edge = edge.to(dev)
    d = delta.to(dtype)
    y = mo.layer_norm(alpha * x.double() + d.double(), w.double(), eps)
    out = torch.empty(n, width, dtype=dtype, device=dev)
    x_out = torch.empty(n, width, device=dev)
    commit = torch.full((6, width), 7.0, device=dev)
    status = torch.zeros(1, dtype=torch.int32, device=dev)
    place = dict(positions=pos, token_rows=trow, token_edges=edge, status=status, eps=eps)
    args = dict(x=x.to(dev), delta=d.to(dev), weight=w.to(dev), alpha=alpha, x_out=x_out)
    dense.residual_norm(out, mix=mix.to(dev), prev=prev.to(dev), commit=commit, **args, **place)
    want, at = [], 0
    for m, c, r in zip(lens, contexts, rows):
        part = y[at:at + m]
        head = prev[r].double() if c else torch.zeros(width, dtype=torch.float64)
        before = torch.cat([head[None], part[:-1]])
        want.append(part + (before - part) * mix.double())
        at += m
    assert rel(x_out, y) < 3e-6
    assert rel(out, torch.cat(want)) < TOL[dtype]
    ends = torch.tensor(lens).cumsum(0) - 1
    assert torch.equal(commit.cpu()[rows], x[ends])
    assert (commit.cpu()[[1, 3, 5]] == 7.0).all()
    dense.residual_norm(out, second_weight=w2.to(dev), **args, **place)
    assert rel(out, mo.layer_norm(y, w2.double(), eps)) < TOL[dtype]
    dense.residual_norm(out, **args, **place)
    assert rel(out, y) < TOL[dtype]
    # fp32 delta next to 16-bit output
    if dtype == torch.bfloat16:
        dense.residual_norm(out, **{**args, "delta": delta.to(dev)}, **place)
        assert rel(x_out, mo.layer_norm(alpha * x.double() + delta.double(), w.double(), eps)) < 3e-6
    assert status.item() == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_residual_norm_embedding_and_decode_rows(dev, dtype):
    g = gen(5)
    vocab, width, n = 50, 40, 6
    table = torch.randn(vocab, width, generator=g).to(dtype).to(dev)
    ids = torch.tensor([3, 49, 0, 7, 7, 1], device=dev)
    mix, prev = torch.rand(width, generator=g).to(dev), torch.randn(n, width, generator=g).to(dev)
    pos = torch.tensor([4, 0, 9, 2, 1, 3], device=dev)
    active = torch.tensor([1, 1, 0, 2, 1, 1], dtype=torch.int32, device=dev)
    out, x = torch.empty(n, width, dtype=dtype, device=dev), torch.empty(n, width, device=dev)
    status = torch.zeros(1, dtype=torch.int32, device=dev)
    place = dict(eps=1e-5, positions=pos, active=active, status=status)
    dense.residual_norm(out, ids=ids, embed=table, x_out=x, mix=mix, prev=prev, **place)
    e = table[ids].double()
    assert torch.equal(x, table[ids].float())
    live = [0, 1, 4, 5]
    before = torch.where((pos > 0)[:, None], prev.double(), torch.zeros_like(e))
    assert rel(out[live], (e + (before - e) * mix.double())[live]) < TOL[dtype]
    # rows that sit out leave their state alone
    commit = torch.full((n, width), 7.0, device=dev)
    w = torch.ones(width, device=dev)
    dense.residual_norm(out, x=x, delta=torch.zeros(n, width, dtype=dtype, device=dev), weight=w, commit=commit, **place)
    assert torch.equal(commit[live], x[live]) and (commit[[2, 3]] == 7.0).all() and status.item() == 0
    # an id outside the table is flagged and reads nothing
    dense.residual_norm(out, ids=torch.full((n,), vocab, device=dev), embed=table, x_out=x, mix=mix, prev=prev, **place)
    assert status.item() == _lib.STATUS_BAD_TOKEN and (x == 0).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [19, 96, 1000, 9000])
def test_poly_norm(dev, dtype, width):
    z = (torch.randn(7, width, generator=gen(width)) * torch.tensor([0.01, 0.1, 1, 1, 2, 5, 20])[:, None]).to(dtype)
    coef = torch.tensor([0.8, -0.6, 0.4, 0.25])
    got = dense.poly_norm(z.to(dev), coef.to(dev), 1e-3)
    want = mo.poly_norm(z.double(), coef.double(), 1e-3)
    for r in range(7):
        assert rel(got[r], want[r]) < TOL[dtype], r
    zz = z.to(dev)
    assert dense.poly_norm(zz, coef.to(dev), 1e-3, out=zz) is zz and torch.equal(zz, got)


# ---- rotation, unit norm, pages ------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,rot,block_size", [
    (4, 2, 32, 48, (16, 1e4, 4.0), 16), (3, 3, 21, 10, None, 4), (8, 1, 64, 128, (64, 500.0, 1.0), 32), (2, 1, 160, 16, (96, 1e5, 2.0), 8),
    (6, 2, 64, 64, (32, 1e4, 3.0), 16), (3, 1, 64, 64, (64, 700.0, 1.0), 32), (5, 5, 128, 128, (128, 1e5, 8.0), 16),
    (4, 2, 128, 128, (48, 1e3, 2.0), 16), (2, 1, 64, 64, None, 16), (2, 1, 64, 64, (24, 1e3, 2.0), 16)])
def test_qk_prepare(dev, dtype, heads, kv_heads, dim, vdim, rot, block_size):
    n, blocks = 9, 8
    g = gen(dim)
    wq, wk, wv = heads * dim, kv_heads * dim, kv_heads * vdim
    x = torch.randn(n, wq + wk + wv, generator=g).to(dtype)
    xd = x.to(dev)
    q, k, v = xd.split([wq, wk, wv], dim=1)
    kp, vp = (PagedKVPool(blocks, kv_heads, block_size, c, dtype, dev) for c in (dim, vdim))
    pos = torch.tensor([0, 1, 2, 50, 333, 4000, 7, 8, 9], device=dev)
    slots = torch.randperm(blocks * block_size, generator=g)[:n].to(dev)
    slots[8] = blocks * block_size  # outside the pool: flagged, nothing written
    status = torch.zeros(1, dtype=torch.int32, device=dev)
    table = None
    if rot is not None:
        from spikeinfer_b200.modeling_manirax import RotaryConfig
        table = RotaryConfig(*rot).table(4001, dev)
    got = dense.qk_prepare(q, k, v, kp, vp, slots, heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, eps=1e-3, rot_table=table,
                           positions=pos, status=status)
    r = None if rot is None else dict(dims=rot[0], base=rot[1], scaling=dict(factor=rot[2]))
    turn = lambda t, c: mo.rms(torch.stack([mo.rotate(t[i].double().view(-1, c), int(pos[i]), r) for i in range(n)]), 1e-3)
    assert rel(got[..., :dim], turn(x[:, :wq], dim)) < TOL[dtype]
    assert (got[..., dim:] == 0).all()
    keep = slots[:8].cpu()
    assert rel(kp.rows()[keep], turn(x[:, wq:wq + wk], dim)[:8]) < TOL[dtype]
    assert torch.equal(vp.rows()[keep].cpu(), x[:8, wq + wk:].view(8, kv_heads, vdim))
    others = torch.ones(blocks * block_size, dtype=torch.bool)
    others[keep] = False
    assert (kp.rows().cpu()[others] == 0).all() and (vp.rows().cpu()[others] == 0).all()
    assert status.item() == _lib.STATUS_BAD_SLOT


# ---- attention -----------------------------------------------------------------------------------------------------
def fill_pool(pool, values, slots):
    """Write ``values [n, heads, dim]`` at flat ``slots`` (pages in the pool's own order)."""
    nb, heads, bs, pad = pool.data.shape
    block, r = slots // bs, slots % bs
    for h in range(heads):
        for d in range(pool.dim):
            if pool.tiled:
                at = (d // 64) * bs * 64 + r * 64 + (((d // 8) % 8) ^ (r & 7)) * 8 + d % 8
            else:
                at = r * pad + d
            pool.data.view(nb, heads, -1)[block, h, at] = values[:, h, d].to(pool.data)


ATTN_SHAPES = {  # heads, kv_heads, dim, vdim, block size
    "d64": (4, 2, 64, 64, 16), "d128": (2, 1, 128, 128, 16), "d64v128": (8, 1, 64, 128, 32), "d128v64": (3, 1, 128, 64, 64),
    "small": (4, 4, 32, 24, 16), "ragged": (5, 1, 80, 100, 16), "group20": (20, 1, 64, 32, 16), "group12": (24, 2, 48, 64, 128),
    "page256": (2, 1, 64, 64, 256), "page8": (2, 1, 64, 64, 8), "page2": (2, 2, 16, 20, 2), "d160": (2, 1, 160, 200, 16),
}


def attention_case(dev, shape, dtype, lens, seed):
    """Sequences of ``lens`` keys in shuffled pages; every page row that holds no key is NaN."""
    heads, kv_heads, dim, vdim, bs = ATTN_SHAPES[shape]
    g = gen(seed)
    need = [-(-m // bs) for m in lens]
    blocks = sum(need) + 2
    pools = [PagedKVPool(blocks, kv_heads, bs, c, dtype, "cpu") for c in (dim, vdim)]
    for p in pools:
        p.data.fill_(float("nan"))
        if p.tiled and p.pad > p.dim:  # padding channels are zero by contract
            p.data.zero_()
            fill_pool(p, torch.full((blocks * bs, kv_heads, p.dim), float("nan")), torch.arange(blocks * bs))
    order = torch.randperm(blocks - 1, generator=g)
    tables = torch.full((len(lens), max(need) + 1), blocks - 1, dtype=torch.int32)
    ks, vs, at = [], [], 0
    for i, m in enumerate(lens):
        tables[i, :need[i]] = order[at:at + need[i]].to(torch.int32)
        at += need[i]
        k = mo.rms(torch.randn(m, kv_heads, dim, generator=g), 1e-5).to(dtype)
        v = torch.randn(m, kv_heads, vdim, generator=g).to(dtype)
        j = torch.arange(m)
        slots = tables[i].long()[j // bs] * bs + j % bs
        fill_pool(pools[0], k, slots)
        fill_pool(pools[1], v, slots)
        ks.append(k)
        vs.append(v)
    for p in pools:
        p.data = p.data.to(dev)
    sizes = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim)
    return pools, tables.to(dev), ks, vs, sizes


def pad_q(q, pool):
    out = torch.zeros(*q.shape[:2], pool.pad, dtype=q.dtype)
    out[..., : q.shape[2]] = q
    return out


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", sorted(ATTN_SHAPES))
def test_sigmoid_attention_portions(dev, shape, dtype):
    """Unequal portions with and without a context, down to one and two tokens, in one call."""
    new, ctx = [1, 2, 70, 130, 37], [0, 300, 0, 127, 16]
    lens = [a + b for a, b in zip(new, ctx)]
    (kp, vp), tables, ks, vs, sizes = attention_case(dev, shape, dtype, lens, 11)
    heads, dim, vdim = sizes["heads"], sizes["dim"], sizes["vdim"]
    g = gen(12)
    bias, scale, out_scale = torch.randn(heads, generator=g) - 2, 0.15, 0.6
    rows = [3, 0, 4, 1, 2]  # portion i is the sequence in row i of `lens`; tables are indexed by row
    tab = torch.empty_like(tables)
    for i, r in enumerate(rows):
        tab[r] = tables[i]
    qs = [mo.rms(torch.randn(m, heads, dim, generator=g), 1e-5).to(dtype) for m in new]
    starts = [sum(new[:i]) for i in range(len(new))]
    plan = PrefillPlan(starts, new, ctx, rows, dev)
    n = sum(new)
    full = torch.full((n, heads * vdim + 5), 9.0, dtype=dtype, device=dev)
    out = full[:, : heads * vdim]
    status = torch.zeros(1, dtype=torch.int32, device=dev)
    dense.sigmoid_attention(pad_q(torch.cat(qs), kp).to(dev), kp, vp, tab, bias.to(dev), out, scale=scale, out_scale=out_scale,
                            plan=plan, status=status, **sizes)
    for i, m in enumerate(new):
        want = out_scale * mo.sigmoid_attention(qs[i].double(), ks[i].double(), vs[i].double(), scale, bias.double())
        assert rel(out[starts[i]:starts[i] + m], want.reshape(m, -1)) < TOL[dtype], i
    assert (full[:, heads * vdim:] == 9.0).all() and status.item() == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", sorted(ATTN_SHAPES))
def test_sigmoid_attention_decode_rows(dev, shape, dtype):
    """Rows of unequal length, one of them inactive, with tables much wider than most rows (several key ranges per row)."""
    lens = [1, 16, 17, 700, 64, 65]
    (kp, vp), tables, ks, vs, sizes = attention_case(dev, shape, dtype, lens, 21)
    heads, dim, vdim = sizes["heads"], sizes["dim"], sizes["vdim"]
    g = gen(22)
    n = len(lens)
    bias, scale = torch.randn(heads, generator=g) - 2, 0.2
    q = mo.rms(torch.randn(n, heads, dim, generator=g), 1e-5).to(dtype)
    active = torch.ones(n, dtype=torch.int32)
    active[4] = _lib.ROW_HELD
    width = 31
    x, w = torch.randn(n, width, generator=g), 1 + 0.1 * torch.randn(width, generator=g)
    gate = torch.randn(n, width, generator=g).to(dtype)
    status = torch.zeros(1, dtype=torch.int32, device=dev)
    out = torch.empty(n, heads * vdim + width, dtype=dtype, device=dev)
    seq, act = torch.tensor(lens, dtype=torch.int32, device=dev), active.to(dev)
    parts = dense.sigmoid_attention(pad_q(q, kp).to(dev), kp, vp, tables, bias.to(dev), out[:, : heads * vdim], scale=scale, out_scale=0.6,
                                    seq_lens=seq, active=act, status=status, partial_sums=True, **sizes)
    assert (parts is not None) == (dtype == torch.bfloat16 and kp.tiled and vp.tiled)
    if parts is not None:
        assert parts.shape[1] > 1
    dense.gated_norm(x.to(dev), w.to(dev), gate.to(dev), out, heads * vdim, eps=1e-4, scale=1.4, partials=parts, left_scale=0.6,
                     seq_lens=seq, active=act)
    for i in range(n):
        if i == 4:
            assert (out[i] == 0).all()
            continue
        want = 0.6 * mo.sigmoid_attention(q[i:i + 1].double(), ks[i].double(), vs[i].double(), scale, bias.double())
        assert rel(out[i, : heads * vdim], want.flatten()) < TOL[dtype], i
        right = 1.4 * mo.rms(x[i].double(), 1e-4) * w.double() * torch.sigmoid(gate[i].double())
        assert rel(out[i, heads * vdim:], right) < TOL[dtype], i
    assert status.item() == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", ["d64", "d128", "ragged", "page256", "d160"])
def test_single_keys_stand_out(dev, shape, dtype):
    """Every weight is almost zero except that of ONE key, for queries whose key sits at a page's, a tile's or a range's
    border, is the query's own, or is the very next one (which must not show)."""
    total = 520
    (kp, vp), tables, ks, vs, sizes = attention_case(dev, shape, dtype, [total], 31)
    heads, kv_heads, dim, vdim = sizes["heads"], sizes["kv_heads"], sizes["dim"], sizes["vdim"]
    k, v = ks[0], vs[0]
    targets = [0, 15, 16, 63, 64, 127, 128, 255, 256, 383, 384, 511, 512, 519]
    bias, scale = torch.full((heads,), -35.0), 62.0 / dim  # a key's product with itself is dim: score 62 - 35
    group = torch.arange(heads) // (heads // kv_heads)
    status = torch.zeros(1, dtype=torch.int32, device=dev)
    sized = dict(scale=scale, status=status, **sizes)
    # prefill: the last query of the portion looks at each target; query j - 1 looks at key j, its future
    q = torch.stack([k[j, group] for j in range(1, total)] + [k[0, group]])        # query i looks at key i + 1
    out = torch.empty(total, heads * vdim, dtype=dtype, device=dev)
    plan = PrefillPlan([0], [total], [0], [0], dev)
    dense.sigmoid_attention(pad_q(q, kp).to(dev), kp, vp, tables, bias.to(dev), out, plan=plan, **sized)
    assert rel(out, mo.sigmoid_attention(q.double(), k.double(), v.double(), scale, bias.double()).reshape(total, -1)) < TOL[dtype]
    for j in targets[1:]:
        assert out[j - 1].abs().max() < 0.2, j      # the next key's weight would be one
    for j in targets:
        q1 = k[j, group][None]
        want = v[j, group].reshape(1, -1)
        got = torch.empty(1, heads * vdim, dtype=dtype, device=dev)
        dense.sigmoid_attention(pad_q(q1, kp).to(dev), kp, vp, tables, bias.to(dev), got,
                                plan=PrefillPlan([0], [1], [total - 1], [0], dev), **sized)
        assert (got.double().cpu() - want.double()).abs().max() < 0.05, j
        for length in (total, j + 1):               # decode: far back, and the newest key itself
            both = torch.empty(1, heads * vdim + 1, dtype=dtype, device=dev)
            seq = torch.tensor([length], dtype=torch.int32, device=dev)
            parts = dense.sigmoid_attention(pad_q(q1, kp).to(dev), kp, vp, tables, bias.to(dev), both[:, :-1], seq_lens=seq,
                                            partial_sums=True, **sized)
            one = torch.ones(1, 1, device=dev)
            dense.gated_norm(one, one[0], one.to(dtype), both, heads * vdim, eps=1e-5, partials=parts, seq_lens=seq)
            assert (both[:, :-1].double().cpu() - want.double()).abs().max() < 0.05, (j, length)
        if j:
            seq = torch.tensor([j], dtype=torch.int32, device=dev)  # one key short: the target is the first it must not see
            parts = dense.sigmoid_attention(pad_q(q1, kp).to(dev), kp, vp, tables, bias.to(dev), both[:, :-1], seq_lens=seq,
                                            partial_sums=True, **sized)
            dense.gated_norm(one, one[0], one.to(dtype), both, heads * vdim, eps=1e-5, partials=parts, seq_lens=seq)
            assert both[:, :-1].abs().max() < 0.2, j
    assert status.item() == 0


def test_bad_tables_and_lengths_are_flagged(dev):
    """A block id outside the pool or a length beyond the table sets a status bit; nothing outside the pool is read."""
    for dtype in DTYPES:
        (kp, vp), tables, ks, vs, sizes = attention_case(dev, "d64", dtype, [40], 41)
        q = torch.ones(1, 4, kp.pad, dtype=dtype, device=dev)
        bias = torch.zeros(4, device=dev)
        out = torch.empty(1, 4 * 64, dtype=dtype, device=dev)
        status = torch.zeros(1, dtype=torch.int32, device=dev)
        bad = tables.clone()
        bad[0, 1] = 10_000
        plan = PrefillPlan([0], [1], [39], [0], dev)
        seq = torch.tensor([40], dtype=torch.int32, device=dev)
        for kw in (dict(plan=plan), dict(seq_lens=seq, partial_sums=True)):
            status.zero_()
            dense.sigmoid_attention(q, kp, vp, bad, bias, out, scale=0.1, status=status, **kw, **sizes)
            assert status.item() & _lib.STATUS_BAD_BLOCK
        status.zero_()
        dense.sigmoid_attention(q, kp, vp, tables, bias, out, scale=0.1, status=status, plan=PrefillPlan([0], [1], [4000], [0], dev), **sizes)
        assert status.item() == _lib.STATUS_BAD_SEQ_LEN and (out == 0).all()
        status.zero_()
        dense.sigmoid_attention(q, kp, vp, tables, bias, out, scale=0.1, status=status, seq_lens=seq * 100, partial_sums=True, **sizes)
        assert status.item() == _lib.STATUS_BAD_SEQ_LEN


# ---- decayed linear attention --------------------------------------------------------------------------------------
DECAY_SHAPES = {"a": (3, 24, 40, (0.5, 0.9, 0.995)), "odd": (2, 13, 11, (1.0, 0.0)), "d64": (2, 64, 64, (0.8, 0.999)),
                "d128": (2, 128, 128, (0.97, 1.0)), "mixed": (1, 128, 64, (0.3,)), "wide": (1, 40, 130, (0.9,)), "narrow": (4, 8, 16, (0.2, 0.4, 0.6, 0.99))}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", sorted(DECAY_SHAPES))
def test_decay_attention_portions_and_steps(dev, shape, dtype):
    """A prompt in portions of 1, 2, 63, 64, 65, 3 and 150 tokens next to a second sequence, then decode steps."""
    heads, dim, vdim, decay = DECAY_SHAPES[shape]
    g = gen(51)
    widths = [heads * dim, heads * dim, heads * vdim]
    portions = [1, 2, 63, 64, 65, 3, 150]
    total, steps = sum(portions), 5
    x = torch.randn(total + steps, sum(widths), generator=g).to(dtype)
    y = torch.randn(total, sum(widths), generator=g).to(dtype)
    act = lambda t: mo.silu(t.double())
    view = lambda t: [p.reshape(t.shape[0], heads, -1) for p in act(t).split(widths, dim=1)]
    want_x, S_x = mo.decay_recurrence(*view(x), list(decay))
    state = torch.full((4, heads, dim, vdim), float("nan"), device=dev)  # slots hold whatever their last owner left
    powers = dense.decay_powers(decay, dev)
    status = torch.zeros(1, dtype=torch.int32, device=dev)
    xd, yd = x.to(dev), y.to(dev)
    at = 0
    tol = 5e-6 if dtype == torch.float32 else TOL[dtype]
    for m in portions:
        both = torch.cat([xd[at:at + m], yd[at:at + m]])
        plan = PrefillPlan([0, m], [m, m], [at, at], [2, 0], dev)
        o = dense.decay_attention(*both.split(widths, dim=1), state, powers, plan=plan, status=status)
        scale = want_x.abs().max()
        assert torch.isfinite(o).all()
        assert float((o[:m].double().cpu() - want_x[at:at + m].reshape(m, -1)).abs().max() / scale) < tol, (at, m)
        at += m
    assert torch.isnan(state[1]).all() and torch.isnan(state[3]).all()
    want_y, S_y = mo.decay_recurrence(*view(y), list(decay))
    assert float((o[150:].double().cpu() - want_y[-150:].reshape(150, -1)).abs().max() / want_y.abs().max()) < tol
    assert rel(state[0], S_y) < tol
    active = torch.tensor([2, 0, 1, 0], dtype=torch.int32, device=dev)
    kept = state[0].clone()
    for i in range(steps):
        rows = xd[total + i].expand(4, -1).contiguous()
        o = dense.decay_attention(*rows.split(widths, dim=1), state, powers, active=active, status=status)
        assert float((o[2].double().cpu() - want_x[total + i].flatten()).abs().max() / want_x.abs().max()) < tol
        assert (o[[0, 1, 3]] == 0).all()
    assert rel(state[2], S_x) < tol and torch.equal(state[0], kept) and torch.isnan(state[1]).all() and status.item() == 0


def test_decay_of_a_long_prompt_keeps_the_first_token(dev):
    """A decay next to one, keys that are zero except the first: the first token's value must still be there at the end."""
    for dtype in DTYPES:
        heads, dim, vdim, n = 1, 64, 64, 1000
        q, k, v = (torch.zeros(n, 64) for _ in range(3))
        k[0] = 1.0
        v[0] = torch.linspace(1, 2, 64)
        q[-1] = 1.0
        state = torch.zeros(1, 1, 64, 64, device=dev)
        d = 0.9995
        x = torch.cat([q, k, v], dim=1).to(dtype).to(dev)
        o = dense.decay_attention(*x.split([64, 64, 64], dim=1), state, dense.decay_powers([d], dev), plan=PrefillPlan([0], [n], [0], [0], dev))
        s1 = mo.silu(torch.tensor(1.0, dtype=torch.float64))
        want = 64 * s1 * s1 * mo.silu(v[0].to(dtype).double()) * d ** (n - 1)
        assert rel(o[-1], want) < (1e-5 if dtype == torch.float32 else 8e-3)


# ---- batch metadata ------------------------------------------------------------------------------------------------
def test_extend_hold_and_resume(dev):
    """Portions pop pages in order, held rows sit out decode steps untouched, freed pages are handed on, and a portion that does
    not fit changes nothing."""
    st = DecodeBatchState(max_rows=3, max_blocks=4, num_blocks=8, block_size=4, device=dev)
    buf = lambda n: (torch.empty(n, dtype=torch.int64, device=dev), torch.empty(n, dtype=torch.int64, device=dev),
                     torch.empty(n, dtype=torch.int32, device=dev), torch.empty(n, dtype=torch.int32, device=dev))
    p, s, r, e = buf(6)
    st.extend(1, 6, p, s, r, e)
    assert p.tolist() == list(range(6)) and s.tolist() == [0, 1, 2, 3, 4, 5] and r.tolist() == [1] * 6 and e.tolist() == [1, 0, 0, 0, 0, 2]
    assert st.seq_lens[1].item() == 6 and st.active[1].item() == _lib.ROW_HELD and st.free_count() == 5
    p, s, r, e = buf(1)
    st.extend(0, 1, p, s, r, e)
    assert s.tolist() == [8] and e.tolist() == [3]
    st.resume(torch.tensor([0], device=dev), torch.tensor([77], device=dev))
    st.advance()
    assert st.seq_lens.tolist() == [2, 6, 1] and st.positions[0].item() == 1 and st.slot_mapping.tolist() == [9, 28, 28]
    assert st.input_ids[0].item() == 77
    p, s, r, e = buf(3)
    st.extend(1, 3, p, s, r, e)  # crosses into a third page
    assert p.tolist() == [6, 7, 8] and s.tolist() == [6, 7, 12] and st.block_tables[1].tolist() == [0, 1, 3, 7]
    st.hold(torch.tensor([0], device=dev))
    before = (st.free_count(), st.block_tables.clone(), st.seq_lens.clone())
    p, s, r, e = buf(8)
    st.extend(1, 8, p, s, r, e)  # 17 tokens: more than the table's four pages
    assert st.status.item() == _lib.STATUS_TABLE_FULL and r.tolist() == [-1] * 8 and s.tolist() == [28] * 8
    st.status.zero_()
    p, s, r, e = buf(14)
    st.extend(2, 14, p, s, r, e)  # four pages, three free
    assert st.status.item() == _lib.STATUS_POOL_EXHAUSTED and st.active[2].item() == 0
    assert st.free_count() == before[0] and torch.equal(st.block_tables, before[1]) and torch.equal(st.seq_lens, before[2])
    st.release(1)
    assert st.free_count() == 6 and st.seq_lens[1].item() == 1
    st.status.zero_()
    st.extend(2, 14, p, s, r, e)
    assert st.status.item() == 0 and st.block_tables[2].tolist() == [3, 1, 0, 4]
