"""GPU: the Gotunex model through the engine (prefill in portions, decode from captured graphs, greedy generation) against the
plain implementation in float64 on the same 16-bit weights."""
from __future__ import annotations

import functools
import json
import os
import subprocess
from pathlib import Path

import numpy as np
import pytest
import torch

import gotunex_cases as gc
from oracle import gotunex_oracle as go
from spikeinfer_b200 import checkpoint, registry
from spikeinfer_b200.modeling_gotunex import GotunexConfig, GotunexModel

pytestmark = pytest.mark.gpu

ROOT = Path(__file__).resolve().parent.parent
DTYPES = [torch.float32, torch.bfloat16]
# rms of the logit difference over the rms of the logits, worst position
TOL = {torch.float32: 2e-5, torch.bfloat16: 3e-2}


@functools.lru_cache(maxsize=None)
def weights(name):
    return go.random_weights(gc.CONFIGS[name], 7)


@functools.lru_cache(maxsize=None)
def reference(name, tokens: tuple):
    layers = []
    return go.forward(list(tokens), go.as_float(weights(name)), gc.CONFIGS[name], layers), layers


def prompt(name, n, seed):
    return torch.randint(0, gc.CONFIGS[name]["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def engine(name, dtype, dev, **kw):
    model = GotunexModel(GotunexConfig.from_dict(gc.CONFIGS[name]), weights(name), device=dev, dtype=dtype)
    args = dict(num_blocks=65, block_size=16, max_num_seqs=4, max_model_len=512)
    args.update(kw)
    return registry.new_engine(model, **args)


def error(got, want) -> float:
    d = got.double().cpu() - want
    return float((d.pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt()).max())


def run(eng, row, tokens):
    """Logits of every token of one portion (or one decode step when the row holds a sequence and one token comes)."""
    if len(tokens) == 1 and row in eng.ledger.seq_lens:
        return eng.feed({row: tokens[0]})
    return eng.model.compute_logits(eng.extend([(row, tokens)]))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(gc.CONFIGS))
def test_whole_prompt_layer_by_layer(dev, name, dtype):
    tokens = prompt(name, 70, 1)
    want, layers = reference(name, tuple(tokens))
    eng = engine(name, dtype, dev)
    got_layers = []
    forward = eng.model.forward_paged
    eng.model.forward_paged = lambda *a: forward(*a, residuals=got_layers)
    logits = run(eng, eng.open_request(), tokens)
    assert len(got_layers) == len(layers)
    for i, (g, w) in enumerate(zip(got_layers, layers)):
        assert error(g, w) < TOL[dtype], f"layer {i}"
    assert error(logits, want) < TOL[dtype]
    eng.state.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(gc.CONFIGS))
def test_token_by_token_equals_the_prompt(dev, name, dtype):
    """The first token alone, then decode steps only (page, chunk and table borders on the way)."""
    tokens = prompt(name, 70, 1)
    want, _ = reference(name, tuple(tokens))
    eng = engine(name, dtype, dev)
    row = eng.open_request()
    for t, tok in enumerate(tokens):
        assert error(run(eng, row, [tok]), want[t:t + 1]) < TOL[dtype], t
    eng.state.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,cuts", [("mixed", [2] * 35), ("odd", [2, 3, 1, 1, 17, 2, 44]), ("wide", [1, 63, 2, 1, 1, 62, 2, 18]),
                                       ("mixed", [64, 2, 64, 20]), ("large_heads", [16, 2, 31, 21]), ("deep", [100, 2, 1, 65, 12]), ("wide", [130, 2, 18])])
def test_portions_of_several_sizes(dev, name, cuts, dtype):
    n = sum(cuts)
    tokens = prompt(name, n, 2)
    want, _ = reference(name, tuple(tokens))
    eng = engine(name, dtype, dev)
    row, at = eng.open_request(), 0
    for c in cuts:
        assert error(run(eng, row, tokens[at:at + c]), want[at:at + c]) < TOL[dtype], at
        at += c
    eng.state.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("block_size", [2, 8, 32])
def test_other_page_sizes(dev, dtype, block_size):
    tokens = prompt("wide", 75, 3)
    want, _ = reference("wide", tuple(tokens))
    eng = engine("wide", dtype, dev, block_size=block_size, num_blocks=512 // block_size)
    row = eng.open_request()
    assert error(run(eng, row, tokens[:67]), want[:67]) < TOL[dtype]
    for t in range(67, 75):
        assert error(run(eng, row, [tokens[t]]), want[t:t + 1]) < TOL[dtype], t
    eng.state.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "wide", "deep"])
def test_unequal_requests_together_and_alone(dev, name, dtype):
    """Portions of unequal requests in one call, decode steps of changing subsets, a row held between portions of its prompt
    while the others decode: each request as if it were alone."""
    lens = [1, 33, 70, 100]
    toks = [prompt(name, n + 12, 10 + i) for i, n in enumerate(lens)]
    want = [reference(name, tuple(t))[0] for t in toks]
    eng = engine(name, dtype, dev)
    rows = [eng.open_request() for _ in lens]
    first = [1, 20, 70, 50]
    logits = eng.model.compute_logits(eng.extend([(r, t[:m]) for r, t, m in zip(rows, toks, first)]))
    at = 0
    for i, m in enumerate(first):
        assert error(logits[at:at + m], want[i][:m]) < TOL[dtype], i
        at += m
    pos = list(first)
    for subset in ([0, 2], [2], [0, 2], [0]):           # 1 and 3 are held between their portions
        got = eng.feed({rows[i]: toks[i][pos[i]] for i in subset})
        for g, i in zip(got, subset):
            assert error(g[None], want[i][pos[i]:pos[i] + 1]) < TOL[dtype], (subset, i)
            pos[i] += 1
    logits = eng.model.compute_logits(eng.extend([(rows[3], toks[3][50:100]), (rows[1], toks[1][20:33])]))
    assert error(logits[:50], want[3][50:100]) < TOL[dtype] and error(logits[50:], want[1][20:33]) < TOL[dtype]
    pos[1], pos[3] = 33, 100
    for _ in range(6):
        got = eng.feed({rows[i]: toks[i][pos[i]] for i in range(4)})
        for i in range(4):
            assert error(got[i][None], want[i][pos[i]:pos[i] + 1]) < TOL[dtype], i
            pos[i] += 1
    eng.state.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_pages_and_slots_used_again(dev, name, dtype):
    """A small pool: requests end, their pages and rows go to the next ones in another order, and nothing of the old ones shows."""
    eng = engine(name, dtype, dev, num_blocks=14, max_num_seqs=2, max_model_len=160)
    a, b, c, d = (prompt(name, n, 20 + n) for n in (120, 60, 100, 33))
    rows = [eng.open_request(), eng.open_request()]
    run(eng, rows[0], a)
    run(eng, rows[1], b[:40])
    with pytest.raises(RuntimeError, match="blocks"):
        eng.extend([(rows[1], prompt(name, 60, 1))])
    eng.release(rows[0])
    row = eng.open_request()
    assert row == rows[0]
    assert error(run(eng, row, c), reference(name, tuple(c))[0]) < TOL[dtype]
    assert error(run(eng, rows[1], b[40:]), reference(name, tuple(b))[0][40:]) < TOL[dtype]
    eng.release(rows[1])
    row = eng.open_request()
    want = reference(name, tuple(d))[0]
    for t in range(len(d)):                             # a fresh one, token by token in the used slot
        assert error(run(eng, row, [d[t]]), want[t:t + 1]) < TOL[dtype], t
    eng.release(row)
    eng.release(rows[0])
    assert eng.state.free_count() == eng.ledger.free == 13
    eng.state.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_over_both_kinds_of_graphs(dev, dtype):
    """A hundred and sixty decoded tokens, from graphs with short tables to those with full ones."""
    name = "wide"
    tokens = prompt(name, 200, 5)
    want, _ = reference(name, tuple(tokens))
    eng = engine(name, dtype, dev, short_context_keys=96)
    assert eng.short_blocks == 6
    row = eng.open_request()
    run(eng, row, tokens[:40])
    for t in range(40, 200):
        assert error(run(eng, row, [tokens[t]]), want[t:t + 1]) < TOL[dtype], t
    assert eng.graphs and eng.short_graphs
    eng.state.check_status()


@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
def test_greedy_generation(dev, name):
    """add_requests + decode_steps in 32 bits pick the plain implementation's tokens; portions of the prompts, eager steps and the
    host-in-the-loop step pick the same."""
    prompts = [prompt(name, n, 40 + n) for n in (3, 29, 17)]
    steps = 14
    w = go.as_float(weights(name))
    want = [go.greedy(p, steps, w, gc.CONFIGS[name]) for p in prompts]

    def generate(**kw):
        eng = engine(name, torch.float32, dev, **kw)
        rows = eng.add_requests(prompts)
        out = [[int(eng.state.next_tokens[r])] for r in rows]
        block = eng.decode_steps(steps - 1)
        for o, r in zip(out, rows):
            o += block[:, r].tolist()
        eng.state.check_status()
        return out

    got = generate()
    for g, (tokens, margins) in zip(got, want):
        for i, (x, y) in enumerate(zip(g, tokens)):
            if x != y:  # only a tie in the plain implementation may be broken differently; what follows differs then
                assert margins[i] < 1e-4, (i, x, y)
                break
    assert generate(max_prefill_tokens=7) == got and generate(use_graph=False) == got
    eng = engine(name, torch.float32, dev)
    rows = eng.add_requests(prompts)
    out = [[int(eng.state.next_tokens[r])] for r in rows]
    host = torch.zeros(4, dtype=torch.int64).pin_memory()
    host.copy_(eng.state.next_tokens.cpu())
    for _ in range(steps - 1):
        host.copy_(eng.step_host(host))
        for o, r in zip(out, rows):
            o.append(int(host[r]))
    assert out == got


def test_snapshot_restores_the_recurrent_state(dev):
    eng = engine("mixed", torch.bfloat16, dev)
    eng.add_requests([prompt("mixed", 20, 1), prompt("mixed", 9, 2)])
    eng.decode_step()
    snap = eng.snapshot()
    first = eng.decode_steps(6).clone()
    eng.restore(snap)
    assert torch.equal(eng.decode_steps(6), first)


def test_feed_forward_beside_the_mixer_changes_nothing(dev):
    tokens = prompt("mixed", 60, 9)
    out = []
    for side in (0, 1 << 20):
        eng = engine("mixed", torch.bfloat16, dev)
        eng.model.side_tokens = side
        row = eng.open_request()
        logits = [run(eng, row, tokens[:41]), run(eng, row, tokens[41:43])]
        logits += [run(eng, row, [t]).clone() for t in tokens[43:]]
        out.append(torch.cat(logits))
    assert torch.equal(*out)


def test_a_shared_cache_is_stored_once(dev):
    eng = engine("mixed", torch.bfloat16, dev)
    layers = eng.cache.layers
    assert layers[2].latent is layers[1].latent is layers[5].latent and layers[3].latent is not layers[1].latent
    pools = {id(x.latent): x.latent.data for x in layers if x.latent is not None}
    states = [t for x in layers for t in x.states.values()]
    assert eng.cache.nbytes == sum(t.numel() * t.element_size() for t in [*pools.values(), *states])


def test_used_slots_and_pages_may_hold_anything(dev):
    """NaN in every state slot and every page: a request that starts at position 0 reads none of it."""
    for dtype in DTYPES:
        eng = engine("mixed", dtype, dev)
        for layer in eng.cache.layers:
            for t in layer.states.values():
                t.fill_(float("nan"))
            if layer.latent is not None:
                layer.latent.data.fill_(float("nan"))
                if layer.latent.tiled:  # padding channels stay zero
                    atoms = layer.latent.data.view(-1, layer.latent.pad // 64, 8, 8, 8)
                    r = torch.arange(8, device=dev)
                    for c in range(layer.latent.pad):
                        if layer.latent.rank <= c < layer.latent.rank_pad or c >= layer.latent.rank_pad + layer.latent.rot_dim:
                            atoms[:, c // 64, r, ((c // 8) % 8) ^ r, c % 8] = 0
        tokens = prompt("mixed", 40, 3)
        want, _ = reference("mixed", tuple(tokens))
        row = eng.open_request()
        assert error(run(eng, row, tokens[:3]), want[:3]) < TOL[dtype]
        assert error(run(eng, row, tokens[3:35]), want[3:35]) < TOL[dtype]
        for t in range(35, 40):
            assert error(run(eng, row, [tokens[t]]), want[t:t + 1]) < TOL[dtype]
        eng.state.check_status()


def test_sums_stay_in_32_bits(dev):
    engine("odd", torch.float32, dev)
    assert not torch.backends.cuda.matmul.allow_tf32 and not torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_program(dev, tmp_path, dtype):
    """bin/trace_run on a model folder: portions, single tokens, requests that end, logits of the wanted places only."""
    name = "mixed"
    cfg = gc.CONFIGS[name]
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    checkpoint.save_safetensors(tmp_path / "model.safetensors", weights(name))
    a, b = prompt(name, 41, 60), prompt(name, 5, 61)
    steps = [dict(step=0, entries=[dict(id="a", tokens=a[:30], want=[0, 29])], end=[]),
             dict(step=1, entries=[dict(id="a", tokens=a[30:32], want=[])], end=[]),
             dict(step=2, entries=[dict(id="a", tokens=a[32:33], want=[0])], end=[]),
             dict(step=3, entries=[dict(id="a", tokens=a[33:], want=[7, 1])], end=["a"]),
             dict(step=4, entries=[dict(id="b", tokens=b[:1], want=[0])], end=[]),
             dict(step=5, entries=[dict(id="b", tokens=b[1:], want=[3])], end=["b"])]
    out = tmp_path / "out"
    out.mkdir()
    r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(tmp_path), "--dtype", dtype, "--out", str(out), "--max-tokens", "48"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=240,
                       env={k: v for k, v in os.environ.items() if k != "SPIKEINFER_B200_LIB"})
    assert r.returncode == 0, r.stderr[-2000:]
    assert [line for line in r.stdout.splitlines() if line.startswith("done")] == [f"done {i}" for i in range(6)]
    assert sorted(p.name for p in out.iterdir()) == ["0.f32", "2.f32", "3.f32", "4.f32", "5.f32"]
    want_a, want_b = reference(name, tuple(a))[0], reference(name, tuple(b))[0]
    tol = TOL[getattr(torch, dtype)]
    for step, want in ((0, want_a[[0, 29]]), (2, want_a[[32]]), (3, want_a[[40, 34]]), (4, want_b[[0]]), (5, want_b[[4]])):
        got = torch.from_numpy(np.fromfile(out / f"{step}.f32", dtype="<f4")).view(-1, cfg["vocab"])
        assert error(got, want) < tol, step
