"""``bench.py --workload manirax``: prefill and decode throughput of the Manirax design beside the spiking model of equal size, and
every kernel of the design against its roofline beside the spiking kernel that plays the same part.

Random weights, synthetic tokens.  Two shapes: ``0.5b`` (24 layers, width 896, 14/2 heads of 64, feed-forward 4864, recurrent
branch 14 x 64 x 64, vocabulary 151,936) and ``7b4`` (four layers of width 3584, 28/4 heads of 128, feed-forward 18,944, recurrent
branch 28 x 128 x 128).  The spiking model has the same layers, width, heads and feed-forward (T = 4).

All times are CUDA events, medians of ``--repeats`` regions after warm-up.  Kernel timings run over enough distinct operand
sets, back to back in one CUDA graph, to exceed L2 (126 MB); the algorithmic bytes count every operand once, flops count
the visible (query, key) pairs once and a weight's pair representation once.
"""
from __future__ import annotations

import json
import statistics
from pathlib import Path

import torch
import torch.nn.functional as F

BF = torch.bfloat16
FALLBACK = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}
SET_BYTES = 300 << 20


def peaks() -> tuple[dict, str]:
    try:
        d = json.loads((Path(__file__).resolve().parent / "MEASURED_PEAKS.json").read_text())
        return {k: float(d[k]) for k in FALLBACK}, "measured"
    except Exception:
        return dict(FALLBACK), "fallback"


def manirax_config(shape: str) -> dict:
    if shape == "0.5b":
        n, width, h, g, d, ff, rh, vocab = 24, 896, 14, 2, 64, 4864, 14, 151936
    else:
        n, width, h, g, d, ff, rh, vocab = 4, 3584, 28, 4, 128, 18944, 28, 32768
    left = dict(heads=h, kv_heads=g, dim=d, vdim=d, scale=d ** -0.5, rot=dict(dims=d, base=1e6))
    right = dict(heads=rh, dim=d, vdim=d, decay=[1 - 2.0 ** -(1 + 8 * i / rh) for i in range(rh)])
    layer = dict(type="parallel", mixer=dict(left=left, right=right, left_scale=1.0, right_scale=1.0), mlp=dict(kind="dense", ff=ff))
    return dict(architecture="Manirax", vocab=vocab, width=width, norm=dict(eps=1e-5), postln_alpha=(2 * n) ** 0.25, layers=[layer] * n)


def manirax_weights(cfg: dict, device, seed: int = 0) -> dict:
    g = torch.Generator(device=device).manual_seed(seed)
    mat = lambda o, i: (torch.randn(o, i, generator=g, device=device) * i ** -0.5).to(BF)
    one = lambda n, v=1.0: torch.full((n,), v, device=device, dtype=BF)
    width = cfg["width"]
    w = {"embed": mat(cfg["vocab"], width), "final.norm": one(width)}
    for i, layer in enumerate(cfg["layers"]):
        p, L, R, ff = f"l{i}.", layer["mixer"]["left"], layer["mixer"]["right"], layer["mlp"]["ff"]
        w.update({p + "norm1": one(width), p + "norm2": one(width), p + "shift": one(width, 0.25)})
        a = p + "mix.left."
        w.update({a + "q": mat(L["heads"] * L["dim"], width), a + "k": mat(L["kv_heads"] * L["dim"], width),
                  a + "v": mat(L["kv_heads"] * L["vdim"], width), a + "pb": one(L["heads"], -5.0), a + "o": mat(width, L["heads"] * L["vdim"])})
        a = p + "mix.right."
        w.update({a + "q": mat(R["heads"] * R["dim"], width), a + "k": mat(R["heads"] * R["dim"], width),
                  a + "v": mat(R["heads"] * R["vdim"], width), a + "g": mat(R["heads"] * R["vdim"], width),
                  a + "norm": one(R["heads"] * R["vdim"]), a + "o": mat(width, R["heads"] * R["vdim"])})
        w.update({p + "mlp.up": mat(ff, width), p + "mlp.down": mat(width, ff),
                  p + "mlp.act": torch.tensor([0.5, 0.3, 0.2, 0.0], device=device, dtype=BF)})
    return w


def build_manirax(shape: str, device):
    from spikeinfer_b200.modeling_manirax import ManiraxConfig, ManiraxModel

    raw = manirax_config(shape)
    return ManiraxModel(ManiraxConfig.from_dict(raw), manirax_weights(raw, device), device=device)


def build_spiking(shape: str, device):
    import bench
    from spikeinfer_b200.modeling import SpikingQwenConfig, SpikingQwenModel

    if shape == "0.5b":
        return bench.build_model(device, seed=0)[1]
    m = manirax_config(shape)
    L = m["layers"][0]
    cfg = SpikingQwenConfig(vocab_size=m["vocab"], hidden_size=m["width"], intermediate_size=L["mlp"]["ff"], num_hidden_layers=len(m["layers"]),
                            num_attention_heads=L["mixer"]["left"]["heads"], num_key_value_heads=L["mixer"]["left"]["kv_heads"],
                            head_dim=L["mixer"]["left"]["dim"])
    return SpikingQwenModel(cfg, bench.random_weights_device(cfg, device, BF, 0), device=device)


def spread(values, digits=2) -> dict:
    return {"median": round(statistics.median(values), digits), "min": round(min(values), digits), "max": round(max(values), digits)}


def event_ms(fn, repeats: int, warmup: int = 3) -> list[float]:
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    out = []
    for _ in range(repeats):
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        a.record()
        fn()
        b.record()
        torch.cuda.synchronize()
        out.append(a.elapsed_time(b))
    return out


def throughput(model, vocab: int, repeats: int, steps: int, prefills, decodes) -> dict:
    """Prefill: (prompts, tokens) groups through the engine's eager call, the first token's logits included.  Decode: (rows, context)
    replays of the captured step."""
    from spikeinfer_b200.registry import new_engine

    out = {"prefill": {}, "decode": {}}
    g = torch.Generator().manual_seed(5)
    for rows, n in prefills:
        eng = new_engine(model, num_blocks=rows * (-(-n // 16) + 1) + 1, block_size=16, max_num_seqs=rows, max_model_len=n + 16)
        prompts = torch.randint(0, vocab, (rows, n), generator=g).tolist()

        def once():
            for r in eng.add_requests(prompts):
                eng.release(r)
        ms = event_ms(once, repeats)
        out["prefill"][f"{rows}x{n}"] = {"ms": spread(ms), "tok_per_s": round(rows * n / statistics.median(ms) * 1e3)}
        del eng
    for rows, ctx in decodes:
        total = ctx + steps * (repeats + 2) + 16
        eng = new_engine(model, num_blocks=rows * (-(-total // 16) + 1) + 1, block_size=16, max_num_seqs=rows, max_model_len=total)
        for s in range(0, rows, 8):
            eng.add_requests(torch.randint(0, vocab, (min(8, rows - s), ctx), generator=g).tolist())
        for _ in range(3):
            eng.decode_step()
        ms = [t / steps for t in event_ms(lambda: [eng.decode_step() for _ in range(steps)], repeats, warmup=0)]
        eng.state.check_status()
        out["decode"][f"{rows}rows_ctx{ctx}"] = {"ms_per_step": spread(ms, 3), "tok_per_s": round(rows / statistics.median(ms) * 1e3)}
        del eng
    torch.cuda.empty_cache()
    return out


def timed_sets(make, nbytes: int, repeats: int) -> list[float]:
    """us per call: ``make()`` returns a closure over operands of its own; enough sets to exceed L2 run back to back in a graph."""
    sets = max(4, min(64, -(-SET_BYTES // max(nbytes, 1))))
    calls = [make() for _ in range(sets)]
    for c in calls:
        c()
    torch.cuda.synchronize()
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.graph(graph):
        for c in calls:
            c()
    inner = 3
    return [t * 1e3 / (sets * inner) for t in event_ms(lambda: [graph.replay() for _ in range(inner)], repeats)]


def entry(us, nbytes, flops, pk) -> dict:
    t = statistics.median(us) * 1e-6
    floor = max(nbytes / (pk["hbm_gbs"] * 1e9), flops / (pk["bf16_tflops"] * 1e12))
    return {"us": spread(us), "MB": round(nbytes / 1e6, 2), "GFLOP": round(flops / 1e9, 2), "roofline_us": round(floor * 1e6, 2),
            "frac": round(floor / t, 3), "bound": "hbm" if nbytes / pk["hbm_gbs"] / 1e9 >= flops / pk["bf16_tflops"] / 1e12 else "tensor"}


def manirax_kernels(shape: str, device, repeats: int, pk: dict) -> dict:
    from spikeinfer_b200.attention import PrefillPlan
    from spikeinfer_b200.engine.kv_state_cache import PagedKVPool
    from spikeinfer_b200.kernels import dense

    cfg = manirax_config(shape)
    L, R = cfg["layers"][0]["mixer"]["left"], cfg["layers"][0]["mixer"]["right"]
    width, ff, H, G, D, RH = cfg["width"], cfg["layers"][0]["mlp"]["ff"], L["heads"], L["kv_heads"], L["dim"], R["heads"]
    rnd = lambda *s: torch.randn(s, device=device).to(BF)
    f32 = lambda *s: torch.randn(s, device=device)
    ones = torch.ones(max(width, RH * D), device=device)
    out = {}

    def add(name, make, nbytes, flops=0):
        out[name] = entry(timed_sets(make, nbytes, repeats), nbytes, flops, pk)

    for kind, n in (("decode64", 64), ("prefill8192", 8192)):
        decode = kind.startswith("decode")
        seqs = 8
        plan = None if decode else PrefillPlan([i * n // seqs for i in range(seqs)], [n // seqs] * seqs, [0] * seqs, list(range(seqs)), device)
        pos = torch.full((n,), 100, device=device) if decode else torch.arange(n // seqs, device=device).repeat(seqs)
        rows = None if decode else (torch.arange(n, device=device, dtype=torch.int32) // (n // seqs)).to(torch.int32)
        edges = None
        if not decode:
            edges = torch.zeros(n, dtype=torch.int32, device=device)
            edges[:: n // seqs] |= 1
            edges[n // seqs - 1:: n // seqs] |= 2
        nstate = 64 if decode else seqs
        active = torch.ones(n, dtype=torch.int32, device=device) if decode else None

        def mk_norm():
            x, xo, d, o, st = f32(n, width), f32(n, width), f32(n, width), rnd(n, width), f32(nstate, width)
            return lambda: dense.residual_norm(o, eps=1e-5, x=x, delta=d, weight=ones[:width], alpha=2.0, x_out=xo, mix=ones[:width], prev=st,
                                               positions=pos, token_rows=rows, token_edges=edges, active=active)
        add(f"residual_norm+shift {kind}", mk_norm, n * width * (4 + 4 + 4 + 2) + (n * width * 4 if decode else 0))

        def mk_poly():
            z, c = rnd(n, ff), ones[:4].clone()
            return lambda: dense.poly_norm(z, c, 1e-5, out=z)
        add(f"poly_norm {kind}", mk_poly, n * ff * 4)

        kp = PagedKVPool(n // 16 + 2, G, 16, D, BF, device)
        vp = PagedKVPool(n // 16 + 2, G, 16, D, BF, device)
        slots = torch.arange(n, device=device)
        table = f32(4096, D // 2, 2)
        W = (H + 2 * G) * D

        def mk_qk():
            q, k, v = rnd(n, W).split([H * D, G * D, G * D], dim=1)
            return lambda: dense.qk_prepare(q, k, v, kp, vp, slots, heads=H, kv_heads=G, dim=D, vdim=D, eps=1e-5, rot_table=table, positions=pos)
        add(f"qk_prepare {kind}", mk_qk, n * W * 4)

        powers = dense.decay_powers(R["decay"], device)

        def mk_decay():
            q, k, v = rnd(n, 3 * RH * D).split([RH * D] * 3, dim=1)
            st = f32(nstate, RH, D, D) * 0.01
            return lambda: dense.decay_attention(q, k, v, st, powers, plan=plan, active=active)
        state_bytes = nstate * RH * D * D * 4
        per_tok = RH * D * (3 * 2 + 4)
        # decode is all state traffic; prefill: the masked product of a 64-token chunk plus the state's two products
        add(f"decay_attention {kind}", mk_decay, n * per_tok + state_bytes * (2 if decode else 1),
            0 if decode else n * RH * (2 * 64 * D + 4 * D * D))

        def mk_gate():
            x, g, o = f32(n, RH * D), rnd(n, RH * D), rnd(n, (H + RH) * D)
            return lambda: dense.gated_norm(x, ones[: RH * D], g, o, H * D, eps=1e-5)
        add(f"gated_norm {kind}", mk_gate, n * RH * D * 8)

    bias = torch.full((H,), -5.0, device=device)
    args = dict(heads=H, kv_heads=G, dim=D, vdim=D, scale=D ** -0.5)
    for rows, keys in ((64, 160), (64, 4096), (256, 4096)):
        nb = rows * -(-keys // 16)
        kv = nb * 16 * G * D * 4
        tables = torch.randperm(nb, device=device, dtype=torch.int32).view(rows, -1)
        lens = torch.full((rows,), keys, dtype=torch.int32, device=device)

        def mk_dec():
            kp, vp = (PagedKVPool(nb, G, 16, D, BF, device) for _ in range(2))
            kp.data.normal_()
            vp.data.normal_()
            q, o = rnd(rows, H, D), rnd(rows, H * D)
            return lambda: dense.sigmoid_attention(q, kp, vp, tables, bias, o, seq_lens=lens, partial_sums=True, **args)
        nbytes = rows * keys * G * D * 4 + rows * H * D * (2 + 4)
        out[f"sigmoid_attention decode {rows}x{keys}"] = entry(timed_sets(mk_dec, max(kv, 5 << 20), repeats), nbytes, 0, pk)
    for seqs, n in ((16, 512), (2, 4096)):
        nb = seqs * n // 16
        kp, vp = (PagedKVPool(nb, G, 16, D, BF, device) for _ in range(2))
        kp.data.normal_()
        vp.data.normal_()
        tables = torch.randperm(nb, device=device, dtype=torch.int32).view(seqs, -1)
        plan = PrefillPlan([i * n for i in range(seqs)], [n] * seqs, [0] * seqs, list(range(seqs)), device)

        def mk_pre():
            q, o = rnd(seqs * n, H, D), rnd(seqs * n, H * D)
            return lambda: dense.sigmoid_attention(q, kp, vp, tables, bias, o, plan=plan, **args)
        nbytes = seqs * n * (2 * H + 2 * G) * D * 2
        out[f"sigmoid_attention prefill {seqs}x{n}"] = entry(timed_sets(mk_pre, nbytes, repeats), nbytes, seqs * n * (n + 1) // 2 * H * 4 * D, pk)
    return out


def spiking_kernels(shape: str, device, repeats: int, pk: dict) -> dict:
    """The spiking model's kernels in the same parts, at the same width, heads and token counts (T = 4)."""
    import bench
    from spikeinfer_b200 import kernels
    from spikeinfer_b200.attention import _causal_offset_mask

    cfg = manirax_config(shape)
    L = cfg["layers"][0]["mixer"]["left"]
    width, ff, H, G, D, T = cfg["width"], cfg["layers"][0]["mlp"]["ff"], L["heads"], L["kv_heads"], L["dim"], 4
    rnd = lambda *s: torch.randn(s, device=device).to(BF)
    out = {}

    def add(name, make, nbytes, flops=0):
        out[name] = entry(timed_sets(make, nbytes, repeats), nbytes, flops, pk)

    for kind, n in (("decode64", 64), ("prefill2048", 2048)):
        def mk_norm():
            h, d, w, o = rnd(T * n, width), rnd(T * n, width), torch.ones(width, device=device, dtype=BF), rnd(T * n, width)
            return lambda: kernels.add_rms_norm(h, d, w, 1e-6, out=o)
        add(f"add_rms_norm {kind}", mk_norm, T * n * width * 8)

        def mk_gate():
            gu = rnd(T, n, 2 * ff)
            beta, th = torch.full((ff,), 0.9, device=device), torch.ones(ff, device=device)
            return lambda: kernels.lif_gate_mul(gu[..., :ff], gu[..., ff:], beta, th)
        add(f"lif_gate_mul {kind}", mk_gate, T * n * ff * 6)

        def mk_qkv():
            qkv = rnd(T, n, (H + 2 * G) * D)
            beta, th = torch.full((D,), 0.9, device=device), torch.ones(D, device=device)
            cos, sin = rnd(n, D), rnd(n, D)
            slots = torch.arange(n, device=device)
            kc, vc = (torch.zeros(T, G, n, D // 32, dtype=torch.int32, device=device) for _ in range(2))
            qp = torch.empty(T, n, H, D // 32, dtype=torch.int32, device=device)
            part = lambda a, b: qkv[..., a * D:b * D].unflatten(-1, (b - a, D))
            S = kernels.LifSiteSpec
            pool = lambda c: dict(packed=c, packed_strides=(c.stride(0), c.stride(2), c.stride(1)), slot_mapping=slots, num_rows=n)
            sites = [S(x=part(0, H), beta=beta, threshold=th, packed=qp, packed_strides=(n * H * D // 32, H * D // 32, D // 32), rope_cos=cos, rope_sin=sin),
                     S(x=part(H, H + G), beta=beta, threshold=th, rope_cos=cos, rope_sin=sin, **pool(kc)),
                     S(x=part(H + G, H + 2 * G), beta=beta, threshold=th, **pool(vc))]
            return lambda: kernels.lif_pack_scatter(sites)
        add(f"lif_qkv_rope_pack_scatter {kind}", mk_qkv, T * n * (H + 2 * G) * D * 2 + T * n * (H + 2 * G) * D // 8)
    for rows, keys in ((64, 160), (64, 4096), (256, 4096)):
        t = bench.time_attention(device, [keys] * rows, -(-keys // 16), 8 if rows > 64 else 24, 3, repeats, hd=D, hq=H, hkv=G)
        out[f"paged_spike_attn decode {rows}x{keys}"] = {"us": t["us_per_call"], "MB": round(t["algorithmic_bytes"] / 1e6, 2),
                                                         "frac": t["frac"], "bound": "hbm"}
    for seqs, n in ((16, 512), (1, 4096)):
        mask = _causal_offset_mask(n, n, device, BF)

        def mk_sdpa():
            q, k, v = rnd(T * seqs, H, n, D), rnd(T * seqs, G, n, D), rnd(T * seqs, G, n, D)
            return lambda: F.scaled_dot_product_attention(q, k, v, attn_mask=mask, enable_gqa=True)
        nbytes = T * seqs * n * (2 * H + 2 * G) * D * 2
        add(f"prefill attention (SDPA on unpacked spikes) {seqs}x{n}", mk_sdpa, nbytes, T * seqs * n * (n + 1) // 2 * H * 4 * D)
    return out


def run(args) -> None:
    import bench

    device = torch.device("cuda", 0)
    torch.cuda.set_device(device)
    pk, source = peaks()
    line = {"workload": "manirax", "data": "synthetic", "dtype": "bf16", "peaks": {**pk, "source": source}, "l2": "operand sets exceed L2",
            "shapes": {}}
    with bench.ClockSampler(0) as clocks:
        for shape in args.manirax_shapes.split(","):
            res = {}
            if not args.manirax_kernels_only:
                for name, build in (("manirax", build_manirax), ("spiking", build_spiking)):
                    model = build(shape, device)
                    res[name] = throughput(model, manirax_config(shape)["vocab"], args.repeats, 16,
                                           ((16, 128), (16, 512), (1, 4096)), ((64, 128), (64, 1024), (1, 128)))
                    del model
                    torch.cuda.empty_cache()
            res["kernels"] = {"manirax": manirax_kernels(shape, device, args.repeats, pk)}
            torch.cuda.empty_cache()
            if not args.manirax_own_only:
                res["kernels"]["spiking"] = spiking_kernels(shape, device, args.repeats, pk)
                torch.cuda.empty_cache()
            line["shapes"][shape] = res
    line["clocks"] = clocks.summary()
    print(json.dumps(line), flush=True)
