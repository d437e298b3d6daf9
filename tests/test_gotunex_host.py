"""Host side of the Gotunex support (no GPU): configuration, registry, layouts, argument structs, and the plain implementation against
closed forms of its mechanisms."""
from __future__ import annotations

import ctypes
import json
import math
import subprocess
from pathlib import Path

import pytest
import torch

import gotunex_cases as gc
from oracle import gotunex_oracle as go
from spikeinfer_b200 import _lib, build, registry
from spikeinfer_b200.attention import PrefillPlan
from spikeinfer_b200.engine.kv_state_cache import LatentSpec, LayerCacheSpec, PagedKVStateCache, PagedLatentPool
from spikeinfer_b200.kernels.experts import operand_tiles, plain_rows
from spikeinfer_b200.modeling_gotunex import (ChannelDeltaConfig, DenseConfig, ExpertsConfig, GotunexConfig, LatentAttentionConfig, _stack)
from spikeinfer_b200.rotary import RotaryConfig

ROOT = Path(__file__).resolve().parent.parent


def changed(name, layer, **kw):
    d = json.loads(json.dumps(gc.CONFIGS[name]))
    d["layers"][layer].update(kw)
    return d


def test_config_reads_every_size_and_constant():
    c = GotunexConfig.from_dict(gc.CONFIGS["mixed"])
    assert (c.vocab, c.width, c.eps, c.embed_scale, len(c.layers)) == (331, 88, 1e-5, 3.5, 6)
    assert c.layers[0].mixer == ChannelDeltaConfig(heads=4, kv_heads=2, dim=24, vdim=40, taps=4)
    assert c.layers[0].mlp == ExpertsConfig(experts=7, top=3, ff=40) and c.layers[1].mlp == DenseConfig(ff=96) and c.layers[3].mlp is None
    assert c.layers[2].mixer == LatentAttentionConfig(heads=5, dim=32, rot_dim=16, vdim=12, q_rank=28, kv_rank=56, scale=0.3,
                                                      rot=RotaryConfig(16, 10000.0), kv_from=1)
    for kw in (dict(type="other"), dict(mlp=dict(kind="sparse"))):
        with pytest.raises(ValueError, match="unknown"):
            GotunexConfig.from_dict(changed("mixed", 1, **kw))
    for src in (0, 2, 5, 7):  # a delta layer, a layer without a cache of its own, itself, one that does not exist
        with pytest.raises(ValueError, match="cache"):
            GotunexConfig.from_dict(changed("mixed", 5, mixer=dict(gc.latent()["mixer"], kv_from=src)))
    with pytest.raises(ValueError, match="share"):
        GotunexConfig.from_dict(changed("mixed", 5, mixer=dict(gc.latent(kv_rank=40)["mixer"], kv_from=1)))
    bad = gc.latent()["mixer"]
    bad["rot"] = dict(bad["rot"], dims=8)
    with pytest.raises(ValueError, match="rotation"):
        GotunexConfig.from_dict(changed("mixed", 1, mixer=bad))
    with pytest.raises(ValueError, match="multiple"):
        GotunexConfig.from_dict(changed("mixed", 0, mixer=gc.delta(heads=3)["mixer"]))


def test_registry_knows_the_design():
    entry = registry.find_model(gc.CONFIGS["odd"])
    assert entry.resolve(entry.config) is GotunexConfig and set(entry.dtypes) == {torch.float32, torch.bfloat16}
    assert entry.components == ("latent",) and entry.engine == "PagedDecodeEngine"
    names = {p.name for p in build.sources(entry.components)}
    assert "spk_latent.cu" in names and "spk_sigmoid_prefill.cu" not in names and "spk_lif.cu" not in names


def test_argument_structs_have_the_header_layout(tmp_path):
    names = {"spk_rms_residual_args": _lib.RmsResidualArgs, "spk_expert_route_args": _lib.ExpertRouteArgs, "spk_experts_args": _lib.ExpertsArgs,
             "spk_latent_prepare_args": _lib.LatentPrepareArgs, "spk_latent_query_args": _lib.LatentQueryArgs,
             "spk_latent_attn_args": _lib.LatentAttnArgs, "spk_latent_out_args": _lib.LatentOutArgs, "spk_delta_args": _lib.DeltaArgs,
             "spk_latent_gather_args": _lib.LatentGatherArgs, "spk_latent_prefill_args": _lib.LatentPrefillArgs}
    lines = [f'printf("{c}.{f} %zu\\n", offsetof({c}, {f}));' for c, s in names.items() for f, _ in s._fields_]
    lines += [f'printf("{c} %zu\\n", sizeof({c}));' for c in names]
    src = tmp_path / "layout.c"
    src.write_text('#include <stddef.h>\n#include <stdio.h>\n#include "spikeinfer_b200.h"\nint main(void){' + "".join(lines) + "return 0;}\n")
    subprocess.run(["gcc", "-I", str(ROOT / "include"), str(src), "-o", str(tmp_path / "layout")], check=True)
    got = dict(line.rsplit(" ", 1) for line in subprocess.run([str(tmp_path / "layout")], check=True, capture_output=True, text=True).stdout.splitlines())
    for c, s in names.items():
        assert int(got[c]) == ctypes.sizeof(s)
        for f, _ in s._fields_:
            assert int(got[f"{c}.{f}"]) == getattr(s, f).offset, (c, f)


def test_host_argument_checks(lib):
    call = lambda name, args: getattr(lib, name)(ctypes.byref(args), None)
    assert lib.spk_rms_residual(None, None) == -4
    a = _lib.RmsResidualArgs(x=1, out1=1, w1=1, n=3, width=0, dtype=_lib.F32)
    assert call("spk_rms_residual", a) == -2
    a.width, a.out1 = 8, None
    assert call("spk_rms_residual", a) == -4
    a.out1, a.w2, a.out2, a.out2_slots, a.out2_top, a.out2_rows, a.out2_tiled = 1, 1, 16, 1, 2, 16, 1
    assert call("spk_rms_residual", a) == -6           # operand tiles hold 16-bit rows
    assert lib.spk_gelu_tanh(1, 1, 3, 2, 4, _lib.F32, None) == -2
    assert lib.spk_expert_rows(0, 2, 4) == 0
    for n, top, experts in ((1, 1, 1), (3, 2, 100), (100, 4, 7)):
        used = min(n * top, experts)
        assert lib.spk_expert_rows(n, top, experts) >= n * top + 7 * used + 256 and lib.spk_expert_rows(n, top, experts) % 8 == 0
    e = _lib.ExpertsArgs(x=16, w=16, out=16, segs=1, rows=12, pairs=4, experts=2, k=8, out_features=8, dtype=_lib.BF16)
    assert call("spk_experts", e) == -3                # rows of an operand matrix come in eights
    p = _lib.LatentPrepareArgs(cq=1, kv=1, ld=8, w_q=1, n=1, q_rank=8, rank=8, rot_dim=3, rank_pad=8, rot_pad=3, block_size=16, num_blocks=2, rot_positions=1)
    assert call("spk_latent_prepare", p) == -2         # an odd rotated part
    t = _lib.LatentAttnArgs(q=1, pool=1, tables=1, partials=1, stats=1, n=1, heads=1, splits=1, num_blocks=1, max_blocks=1, rank=8, rot_dim=2, rank_pad=8,
                            rot_pad=2, block_size=16, table_rows=1)
    assert call("spk_latent_attn", t) == -4            # neither lengths nor positions
    d = _lib.DeltaArgs(n=1, heads=3, kv_heads=2, dim=4, vdim=4, taps=4, state_rows=1)
    assert call("spk_delta_step", d) == -2
    assert lib.spk_latent_attn_splits(_lib.F32, 64, 16, 64, 16, 0, 16, 1, 4, 100) == 1


def test_operand_tiles_are_the_swizzle():
    w = torch.arange(16 * 100, dtype=torch.float32).view(16, 100)
    t = operand_tiles(w)
    assert t.shape == (2, 16, 64) and torch.equal(plain_rows(t, 100), w)
    for r, c in ((0, 0), (5, 99), (15, 64), (9, 63)):
        assert t[c // 64, r, (((c // 8) % 8) ^ (r & 7)) * 8 + c % 8] == w[r, c]
    assert (plain_rows(t, 128)[:, 100:] == 0).all()


def test_parts_of_a_stacked_projection_start_at_multiples_of_eight():
    parts = {"a": torch.ones(3, 5), "b": torch.full((8, 5), 2.0), "c": torch.full((9, 5), 3.0)}
    w, at = _stack(parts)
    assert w.shape == (32, 5) and all(s.start % 8 == 0 for s in at.values())
    for name, part in parts.items():
        assert torch.equal(w[at[name]], part)
    assert w.sum() == sum(p.sum() for p in parts.values())


def test_latent_pools_and_sharing():
    pool = PagedLatentPool(3, 16, 56, 16, torch.bfloat16, "cpu")
    assert pool.tiled and (pool.rank_pad, pool.rot_pad, pool.pad) == (64, 64, 128)
    plain = PagedLatentPool(3, 16, 56, 16, torch.float32, "cpu")
    assert not plain.tiled and plain.pad == 72 and plain.rows().shape == (48, 72)
    pool.data.view(3, -1)[1, 8 * 128 + 512 + 5 * 64 + ((1 ^ 5) << 3) + 2] = 7.0     # page 1, row 13, rotated channel 10
    assert pool.rows()[16 + 13, 56 + 10] == 7.0
    specs = [LayerCacheSpec(states=(("s", (2, 3)),)), LayerCacheSpec(latent=LatentSpec(8, 4)), LayerCacheSpec(latent_from=1)]
    cache = PagedKVStateCache(specs, 4, 16, 2, torch.float32, "cpu")
    assert cache.layers[2].latent is cache.layers[1].latent and cache.nbytes == 4 * (2 * 6 + 4 * 16 * 12)
    for src in (0, 2):
        with pytest.raises(ValueError, match="share"):
            PagedKVStateCache([specs[0], specs[1], LayerCacheSpec(latent_from=src)], 4, 16, 2, torch.float32, "cpu")


def test_portion_table():
    plan = PrefillPlan([0, 5, 7], [5, 2, 40], [0, 31, 8], [3, 0, 1], torch.device("cpu"))
    assert plan.portions().tolist() == [[0, 5, 3, 0], [5, 2, 0, 31], [7, 40, 1, 8]] and plan.most_keys == 48
    starts, total, rows = plan.contexts()
    assert (starts, total) == ([0, 5, 38], 86)
    assert rows.tolist() == [[0, 5, 3, 0], [5, 16, 0, 0], [21, 16, 0, 16], [37, 1, 0, 32], [38, 16, 1, 0], [54, 16, 1, 16], [70, 16, 1, 32]]
    assert sorted(plan.context_tiles(32).tolist()) == [[0, 5, 0, 0], [5, 2, 5, 31], [7, 32, 38, 8], [39, 8, 38, 40]]


# ---- the plain implementation itself ---------------------------------------------------------------------------
def test_oracle_mechanisms_against_closed_forms():
    g = torch.Generator().manual_seed(1)
    rnd = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    # no decay and unit keys that repeat: after a write of strength one the state returns exactly the last value
    k = torch.nn.functional.normalize(rnd(1, 6), dim=1).expand(5, 6)
    v = rnd(5, 3)
    o, S = go.delta_rule(k, k, v, torch.ones(5, dtype=torch.float64), torch.zeros(5, 6, dtype=torch.float64))
    assert torch.allclose(o, v) and torch.allclose(S.t() @ k[0], v[-1])
    # orthogonal keys: plain decayed sums, the read-out sees the current write
    q, beta, ld = rnd(4, 4), torch.rand(4, generator=g, dtype=torch.float64), -torch.rand(4, 4, generator=g, dtype=torch.float64)
    k = torch.eye(4, dtype=torch.float64)
    o, _ = go.delta_rule(q, k, v[:4], beta, ld)
    for t in range(4):
        want = sum(q[t, s] * torch.exp(ld[s + 1: t + 1, s].sum()) * beta[s] * v[s] for s in range(t + 1))
        assert torch.allclose(o[t], want)
    x, taps = rnd(7, 3), rnd(3, 4)
    want = torch.nn.functional.conv1d(x.t()[None], taps[:, None], padding=3, groups=3)[0, :, :7].t()
    assert torch.allclose(go.causal_conv(x, taps), want)
    assert torch.allclose(go.softplus(x * 30), torch.nn.functional.softplus(x * 30, threshold=1000))
    assert torch.allclose(go.gelu_tanh(x), torch.nn.functional.gelu(x, approximate="tanh"))
    rot = dict(dims=6, base=100.0)
    a, b = rnd(8), rnd(8)
    dot = lambda p, s: (go.rotate(a, p, rot) * go.rotate(b, s, rot)).sum()
    assert torch.allclose(dot(17, 5), dot(29, 17)) and torch.equal(go.rotate(a, 9, rot)[6:], a[6:])
    s = rnd(5)
    p = go.sink_softmax(s, torch.tensor(0.3, dtype=torch.float64))
    assert torch.allclose(p, torch.softmax(torch.cat([s, torch.tensor([0.3])]), 0)[:5])
    assert torch.allclose(go.sink_softmax(s + 800, torch.tensor(-800.0, dtype=torch.float64)).sum(), torch.ones((), dtype=torch.float64))
    # scores of keys spelled out equal scores of queries taken into the latent space
    c, w, qn = rnd(9, 12), rnd(5, 12), rnd(5)
    assert torch.allclose((c @ w.t()) @ qn, c @ (w.t() @ qn))
    cfg = dict(router=dict(experts=2, top=1))
    ew = {f"e{e}.{n}": rnd(*shape) for e in range(2) for n, shape in (("gate", (4, 3)), ("up", (4, 3)), ("down", (3, 4)))}
    ew["table"] = torch.tensor([[1], [0]])
    h = rnd(2, 3)
    one = lambda x, e: (go.silu(x @ ew[f"e{e}.gate"].t()) * (x @ ew[f"e{e}.up"].t())) @ ew[f"e{e}.down"].t()
    assert torch.allclose(go.table_experts(h, [1, 0], ew, "", cfg), torch.stack([one(h[0], 0), one(h[1], 1)]))


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_oracle_is_causal(name):
    cfg = gc.CONFIGS[name]
    w = go.as_float(go.random_weights(cfg, 3))
    tokens = torch.randint(0, cfg["vocab"], (12,), generator=torch.Generator().manual_seed(4)).tolist()
    full = go.forward(tokens, w, cfg)
    assert torch.allclose(go.forward(tokens[:7], w, cfg), full[:7]) and full.shape == (12, cfg["vocab"])
    tokens[8] = (tokens[8] + 1) % cfg["vocab"]
    other = go.forward(tokens, w, cfg)
    assert torch.allclose(other[:8], full[:8]) and (other[8:] - full[8:]).abs().amax(-1).min() > 1e-3


@pytest.mark.parametrize("part", ["mix.sink", "mix.A_log", "mix.dt_bias", "mix.k.conv", "mlp.table", "mix.dkv.norm"])
def test_every_mechanism_shows_in_the_logits(part):
    """A change of one mechanism's parameters moves the logits by far more than the tests' tolerances."""
    cfg = gc.CONFIGS["mixed"]
    w = go.random_weights(cfg, 3)
    tokens = torch.randint(0, cfg["vocab"], (20,), generator=torch.Generator().manual_seed(4)).tolist()
    want = go.forward(tokens, go.as_float(w), cfg)
    for k in [k for k in w if k.endswith(part)]:
        w[k] = w[k].flip(0) if part == "mlp.table" else w[k] + 1
    got = go.forward(tokens, go.as_float(w), cfg)
    assert float((got - want).pow(2).mean().sqrt() / want.pow(2).mean().sqrt()) > 0.06
    assert math.isfinite(float(got.sum()))
