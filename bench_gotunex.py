"""``bench.py --workload gotunex``: prefill and decode throughput of the Gotunex design beside Manirax (the closest design the engine
serves) of equal size, and every kernel of the design against its roofline beside the Manirax kernel that plays the same part.

Random weights, synthetic tokens.  Two shapes, layers, width, heads, head size and vocabulary those of ``bench_manirax.py``: ``0.5b`` (24
layers, width 896, 14 heads of 64) and ``7b4`` (four layers, width 3584, 28 heads of 128).  Layers alternate between channel delta and latent
attention, every second latent layer reads its predecessor's cache; the first layer has a dense feed-forward of Manirax's size, the others
16 experts of which a token uses two.

Timing as in ``bench_manirax.py``: CUDA events, medians, operand sets beyond L2.  Algorithmic bytes count every operand once; the flops of
an attention count visible (query, key) pairs in the cheaper of the two forms (keys and values spelled out for prefill)."""
from __future__ import annotations

import json

import torch
import torch.nn.functional as F

from bench_manirax import (BF, build_manirax, entry, manirax_config, manirax_kernels, peaks, throughput, timed_sets)


def gotunex_config(shape: str) -> dict:
    m = manirax_config(shape)
    L = m["layers"][0]
    width, heads, d, ff = m["width"], L["mixer"]["left"]["heads"], L["mixer"]["left"]["dim"], L["mlp"]["ff"]
    rot_dim, q_rank, kv_rank = (32, 384, 256) if shape == "0.5b" else (64, 1536, 512)
    moe = dict(kind="moe", router=dict(experts=16, top=2), expert=dict(ff=ff // 4))
    layers, owner = [], None
    for i in range(len(m["layers"])):
        mlp = dict(kind="dense", ff=ff) if i == 0 else moe
        if i % 2 == 0:
            layers.append(dict(type="channel_delta", mixer=dict(heads=heads, kv_heads=heads, dim=d, vdim=d, conv=4), mlp=mlp))
            continue
        mixer = dict(heads=heads, dim=d, rot_dim=rot_dim, vdim=d, q_rank=q_rank, kv_rank=kv_rank, scale=(d + rot_dim) ** -0.5,
                     rot=dict(base=1e6, dims=rot_dim))
        if owner is not None:
            mixer["kv_from"], owner = owner, None
        else:
            owner = i
        layers.append(dict(type="latent_attention", mixer=mixer, mlp=mlp))
    return dict(architecture="Gotunex", vocab=m["vocab"], width=width, norm=dict(eps=1e-5), embedding=dict(scale=width ** 0.5), layers=layers)


def gotunex_weights(cfg: dict, device, seed: int = 0) -> dict:
    g = torch.Generator(device=device).manual_seed(seed)
    mat = lambda o, i: (torch.randn(o, i, generator=g, device=device) * i ** -0.5).to(BF)
    one = lambda n, v=1.0: torch.full((n,), v, device=device, dtype=BF)
    width, vocab = cfg["width"], cfg["vocab"]
    w = {"embed": (torch.randn(vocab, width, generator=g, device=device) / cfg["embedding"]["scale"]).to(BF), "final.norm": one(width),
         "head": mat(vocab, width)}
    for i, layer in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", layer["mixer"], layer["mlp"]
        a, b = p + "mix.", p + "mlp."
        w.update({p + "norm1": one(width), p + "norm2": one(width)})
        if layer["type"] == "channel_delta":
            H, G, D, V, T, r = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"], m["dim"]
            for name, rows in (("q", G * D), ("k", G * D), ("v", H * V)):
                w[a + name], w[a + name + ".conv"] = mat(rows, width), one(rows * T, 0.4).view(rows, T)
            w.update({a + "b": mat(H, width), a + "A_log": one(H, 0.0), a + "dt_bias": one(H * D, -3.0), a + "a1": mat(r, width), a + "a2": mat(H * D, r),
                      a + "g1": mat(r, width), a + "g2": mat(H * V, r), a + "norm": one(V), a + "o": mat(width, H * V)})
        else:
            H, D, R, V, K, Q = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"]
            w.update({a + "dq": mat(Q, width), a + "dq.norm": one(Q), a + "uq": mat(H * (D + R), Q), a + "uk": mat(H * D, K), a + "uv": mat(H * V, K),
                      a + "sink": one(H, 0.0), a + "g": mat(H * V, width), a + "o": mat(width, H * V)})
            if m.get("kv_from") is None:
                w.update({a + "dkv": mat(K + R, width), a + "dkv.norm": one(K)})
        if mlp["kind"] == "dense":
            w.update({b + "up": mat(mlp["ff"], width), b + "down": mat(width, mlp["ff"])})
        else:
            E, top, ff = mlp["router"]["experts"], mlp["router"]["top"], mlp["expert"]["ff"]
            for e in range(E):
                w.update({f"{b}e{e}.gate": mat(ff, width), f"{b}e{e}.up": mat(ff, width), f"{b}e{e}.down": mat(width, ff)})
            w[b + "table"] = torch.rand(vocab, E, generator=g, device=device).topk(top).indices.to(torch.int32)
    return w


def build_gotunex(shape: str, device):
    from spikeinfer_b200.modeling_gotunex import GotunexConfig, GotunexModel

    raw = gotunex_config(shape)
    return GotunexModel(GotunexConfig.from_dict(raw), gotunex_weights(raw, device), device=device)


def gotunex_kernels(shape: str, device, repeats: int, pk: dict, only=()) -> dict:
    from spikeinfer_b200.attention import PrefillPlan
    from spikeinfer_b200.engine.kv_state_cache import PagedLatentPool
    from spikeinfer_b200.kernels import delta, dense, experts, latent

    cfg = gotunex_config(shape)
    lat, dm = cfg["layers"][1]["mixer"], cfg["layers"][0]["mixer"]
    moe, ff = cfg["layers"][1]["mlp"], cfg["layers"][0]["mlp"]["ff"]
    width, H, D, R, V, K, Q = (cfg["width"], *(lat[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank")))
    E, top, fe = moe["router"]["experts"], moe["router"]["top"], moe["expert"]["ff"]
    rnd = lambda *s: torch.randn(s, device=device).to(BF)
    f32 = lambda *s: torch.randn(s, device=device)
    ones = torch.ones(max(width, Q, K, ff), device=device)
    out = {}

    def add(name, make, nbytes, flops=0, at_least=0):
        if not only or any(name.startswith(o) for o in only):
            out[name] = entry(timed_sets(make, max(nbytes, at_least), repeats), nbytes, flops, pk)

    table = torch.rand(4096, E, device=device).topk(top).indices.to(torch.int32)
    part = lambda o, i: [rnd(o, i) * i ** -0.5 for _ in range(E)]
    sets = 4 if shape == "0.5b" else 1  # a 7b4 set of experts is beyond L2 by itself
    weights = [experts.ExpertWeights(part(fe, width), part(fe, width), part(width, fe), table) for _ in range(sets)]
    rot = f32(8192, R // 2, 2)
    for kind, n in (("decode64", 64), ("prefill8192", 8192)):
        decode = kind.startswith("decode")
        seqs = 8
        plan = None if decode else PrefillPlan([i * n // seqs for i in range(seqs)], [n // seqs] * seqs, [0] * seqs, list(range(seqs)), device)
        pos = torch.full((n,), 100, device=device) if decode else torch.arange(n // seqs, device=device).repeat(seqs)
        ids = torch.randint(0, 4096, (n,), device=device)
        router = experts.ExpertRouter(weights, 4096)
        routes = router(ids)
        nstate = 64 if decode else seqs
        active = torch.ones(n, dtype=torch.int32, device=device) if decode else None
        add(f"route {kind} ({len(weights)} layers)", lambda: lambda: router(ids), n * top * 8 * len(weights))

        def mk_norm():
            x, d, h, p, xs = f32(n, width), f32(n, width), rnd(n, width), f32(weights[0].rows(n), width), weights[0].sorted_matrix(n, width)
            return lambda: dense.rms_residual(eps=1e-5, x=x, delta=d, x_out=x, pairs=p, pair_slots=routes[0].slots, pair_scale=0.5, w1=ones[:width],
                                              out1=h, w2=ones[:width], out2=xs, out2_slots=routes[0].slots, out2_tiled=True)
        add(f"rms_residual {kind}", mk_norm, n * width * (4 + 4 + 4 + 2 + top * (4 + 2)))

        def mk_gelu():
            z, o = rnd(n, ff), rnd(n, ff)
            return lambda: dense.gelu_tanh(z, o)
        add(f"gelu {kind}", mk_gelu, n * ff * 4)
        state = {"i": 0}

        def mk_experts():
            i = state["i"] = (state["i"] + 1) % len(weights)
            xs = weights[i].sorted_matrix(n, width)
            xs.normal_()
            return lambda: experts.experts_forward(xs, weights[i], routes[i])
        used = min(E, n * top)
        add(f"experts {kind}", mk_experts, used * 3 * fe * width * 2 + n * top * (width * 6 + fe * 4), n * top * 6 * width * fe)

        pool = PagedLatentPool(n // 16 + 2, 16, K, R, BF, device)
        slots = torch.arange(n, device=device)

        def mk_prepare():
            z = rnd(n, Q + K + R)
            return lambda: latent.latent_prepare(z[:, :Q], ones[:Q], eps=1e-5, kv=z[:, Q:], w_kv=ones[:K], pool=pool, rot_table=rot, positions=pos,
                                                 slot_mapping=slots)
        add(f"latent_prepare {kind}", mk_prepare, n * (Q + K + R) * 4)
        if decode:
            def mk_query():
                q, wk = rnd(n, H * (D + R)), rnd(H * D, K)
                return lambda: latent.latent_query(q, wk, pool, rot, pos, heads=H, dim=D)
            add(f"latent_query {kind}", mk_query, n * H * (D + R + K + R) * 2 + H * D * K * 2, n * H * D * K * 2)
        G = dm["kv_heads"]
        DH, DD, DV, T = dm["heads"], dm["dim"], dm["vdim"], dm["conv"]
        widths = [G * DD, G * DD, DH * DV, DH]
        conv = [f32(c, T) for c in widths[:3]]
        a_log, dt, nw = torch.zeros(DH, device=device), torch.full((DH * DD,), -3.0, device=device), ones[:DV]

        def mk_delta():
            z, y, o = rnd(n, -(-sum(widths) // 8) * 8), rnd(n, DH * (DD + DV)), rnd(n, DH * DV)
            st, cs = f32(nstate, DH, DD, DV) * 0.01, f32(nstate, T, sum(widths[:3]))
            where = dict(positions=pos, active=active) if decode else dict(plan=plan)
            return lambda: delta.delta_rule(*z[:, : sum(widths)].split(widths, dim=1), *y.split([DH * DD, DH * DV], dim=1), conv=conv, a_log=a_log, dt_bias=dt,
                                            norm=nw, state=st, conv_state=cs, out=o, kv_heads=G, eps=1e-5, **where)
        per_tok = (sum(widths) + DH * (DD + 2 * DV)) * 2
        add(f"delta_rule {kind}", mk_delta, n * per_tok + nstate * DH * DD * DV * 4 * (2 if decode else 1) + (nstate * T * sum(widths[:3]) * 4 if decode else 0),
            0 if decode else n * DH * (2 * 2 * 64 * DD + 64 * DV * 2 + 6 * DD * DV))

    sink = torch.zeros(H, device=device)
    w_uv = rnd(H * V, K) * K ** -0.5
    for rows, keys in ((64, 160), (64, 4096), (256, 4096)):
        nb = rows * -(-keys // 16)
        tables = torch.randperm(nb, device=device, dtype=torch.int32).view(rows, -1)
        lens = torch.full((rows,), keys, dtype=torch.int32, device=device)

        def mk_dec():
            pool = PagedLatentPool(nb, 16, K, R, BF, device)
            pool.data.normal_()
            q, g, o = rnd(rows, H, pool.pad), rnd(rows, H * V), rnd(rows, H * V)
            return lambda: latent.latent_attention(q, pool, tables, sink, w_uv, g, o, vdim=V, scale=0.02, seq_lens=lens)
        nbytes = rows * keys * (K + R) * 2 + rows * H * (K + R + 2 * V) * 2 + H * V * K * 2
        add(f"latent_attention decode {rows}x{keys}", mk_dec, nbytes, rows * keys * H * (4 * K + 2 * R), 5 << 20)
    for seqs, n in ((16, 512), (2, 4096)):
        nb = seqs * n // 16
        pool = PagedLatentPool(nb, 16, K, R, BF, device)
        pool.data.normal_()
        tables = torch.randperm(nb, device=device, dtype=torch.int32).view(seqs, -1)
        plan = PrefillPlan([i * n for i in range(seqs)], [n] * seqs, [0] * seqs, list(range(seqs)), device)
        pos = torch.arange(n, device=device).repeat(seqs)
        rows = (torch.arange(seqs * n, device=device) // n).to(torch.int32)
        w_uk = rnd(H * D, K) * K ** -0.5
        w_kv = latent.spelled_out_weights(w_uk, w_uv, H)

        def mk_pre():
            q, g, o = rnd(seqs * n, H * (D + R)), rnd(seqs * n, H * V), rnd(seqs * n, H * V)
            return lambda: latent.latent_prefill(q, pool, tables, w_uk, w_uv, w_kv, sink, g, o, rot_table=rot, positions=pos, token_rows=rows, plan=plan, heads=H, dim=D,
                                                 vdim=V, scale=0.07)
        nbytes = seqs * n * (H * (D + R + 2 * V) + K + R) * 2
        add(f"latent_attention prefill {seqs}x{n}", mk_pre, nbytes, seqs * n * (n + 1) // 2 * H * 2 * (D + R + V) + seqs * n * H * 2 * K * (D + V))
    return out


def library_kernels(shape: str, device, repeats: int, pk: dict) -> dict:
    """The products Manirax leaves to the library in the place of the experts: its dense feed-forward's two GEMMs."""
    m = manirax_config(shape)
    width, ff = m["width"], m["layers"][0]["mlp"]["ff"]
    rnd = lambda *s: torch.randn(s, device=device).to(BF)
    out = {}
    for kind, n in (("decode64", 64), ("prefill8192", 8192)):
        def mk():
            x, u, d = rnd(n, width), rnd(ff, width), rnd(width, ff)
            return lambda: torch.mm(F.linear(x, u), d.t(), out_dtype=torch.float32)
        nbytes = 4 * ff * width + n * (6 * width + 4 * ff)
        out[f"feed-forward GEMMs {kind}"] = entry(timed_sets(mk, nbytes, repeats), nbytes, 4 * n * ff * width, pk)
    return out


def run(args) -> None:
    import bench

    device = torch.device("cuda", 0)
    torch.cuda.set_device(device)
    pk, source = peaks()
    line = {"workload": "gotunex", "data": "synthetic", "dtype": "bf16", "peaks": {**pk, "source": source}, "l2": "operand sets exceed L2", "shapes": {}}
    only = tuple(x for x in args.gotunex_only.split(",") if x)
    with bench.ClockSampler(0) as clocks:
        for shape in args.gotunex_shapes.split(","):
            res = {}
            if not args.gotunex_kernels_only:
                for name, build in (("gotunex", build_gotunex), *(() if args.gotunex_own_only else (("manirax", build_manirax),))):
                    model = build(shape, device)
                    res[name] = throughput(model, manirax_config(shape)["vocab"], args.repeats, 16, ((16, 128), (16, 512), (1, 4096)),
                                           ((64, 128), (64, 1024), (1, 128)))
                    del model
                    torch.cuda.empty_cache()
            res["kernels"] = {"gotunex": gotunex_kernels(shape, device, args.repeats, pk, only)}
            torch.cuda.empty_cache()
            if not args.gotunex_own_only:
                res["kernels"]["manirax"] = {**manirax_kernels(shape, device, args.repeats, pk), **library_kernels(shape, device, args.repeats, pk)}
                torch.cuda.empty_cache()
            line["shapes"][shape] = res
    line["clocks"] = clocks.summary()
    print(json.dumps(line), flush=True)
