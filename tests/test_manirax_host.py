"""Host side of the Manirax support (no GPU): configuration, registry, checkpoint files, portions and their ledger, work lists,
and the plain implementation against closed forms of its mechanisms."""
from __future__ import annotations

import ctypes
import json
import subprocess
from pathlib import Path

import pytest
import torch

import manirax_cases as mc
from oracle import manirax_oracle as mo
from spikeinfer_b200 import _lib, build, checkpoint, registry
from spikeinfer_b200.attention import PrefillPlan
from spikeinfer_b200.engine.block_ledger import BlockLedger, cut_portions
from spikeinfer_b200.engine.kv_state_cache import PagedKVPool
from spikeinfer_b200.modeling_manirax import ManiraxConfig, RotaryConfig

ROOT = Path(__file__).resolve().parent.parent


def test_config_reads_every_size_and_constant():
    c = ManiraxConfig.from_dict(mc.CONFIGS["mixed"])
    assert (c.vocab, c.width, c.eps, c.alpha, len(c.layers)) == (331, 72, 1e-5, 1.7, 3)
    a, b, d = c.layers
    assert (a.left.heads, a.left.kv_heads, a.left.dim, a.left.vdim, a.left.scale) == (4, 2, 32, 32, 0.2)
    assert a.left.rot == RotaryConfig(16, 10000.0, 4.0) and b.left.rot.factor == 1.0
    assert a.right.decay == (0.5, 0.9, 0.995) and (a.right.dim, a.right.vdim) == (24, 40)
    assert (a.left_scale, a.right_scale, a.ff, b.ff) == (0.7, 1.3, 80, None)
    odd = ManiraxConfig.from_dict(mc.CONFIGS["odd"])
    assert odd.layers[0].left.rot is None and odd.layers[1].left.rot.factor == 1.0
    for key, value in (("type", "other"), ("mlp", dict(kind="sparse", ff=3))):
        bad = json.loads(json.dumps(mc.CONFIGS["mixed"]))
        bad["layers"][0][key] = value
        with pytest.raises(ValueError, match="unknown"):
            ManiraxConfig.from_dict(bad)
    bad = json.loads(json.dumps(mc.CONFIGS["mixed"]))
    bad["layers"][0]["mixer"]["right"]["decay"] = [0.5]
    with pytest.raises(ValueError, match="decay"):
        ManiraxConfig.from_dict(bad)


def test_registry_finds_model_classes_by_config():
    entry = registry.find_model(mc.CONFIGS["odd"])
    assert entry.resolve(entry.config) is ManiraxConfig and entry.resolve(entry.model).__name__ == "ManiraxModel"
    for d in ({"architecture": "SpikingQwen"}, {"architectures": ["FastSpikingQwenForCausalLM"]}):
        spiking = registry.find_model(d)
        cfg = spiking.resolve(spiking.config).from_dict(dict(vocab_size=64, hidden_size=32, intermediate_size=48, num_hidden_layers=1,
                                                             num_attention_heads=4, num_key_value_heads=2, unrelated=1))
        assert cfg.head_dim == 8 and cfg.T == 4
    with pytest.raises(ValueError, match="unknown architecture"):
        registry.find_model({"architecture": "Nothing"})


def test_safetensors_round_trip(tmp_path):
    g = torch.Generator().manual_seed(0)
    tensors = {"a": torch.randn(3, 5, generator=g).to(torch.bfloat16), "b": torch.randn(7, generator=g),
               "c": torch.arange(3, dtype=torch.int32), "empty": torch.empty(0, 4), "d": torch.randn(1, generator=g).to(torch.bfloat16)}
    checkpoint.save_safetensors(tmp_path / "model.safetensors", tensors)
    got = checkpoint.load_weights(tmp_path)
    assert set(got) == set(tensors)
    for k, t in tensors.items():
        assert got[k].dtype == t.dtype and torch.equal(got[k], t), k
    # shards named by an index
    checkpoint.save_safetensors(tmp_path / "x.safetensors", {"a": tensors["a"]})
    checkpoint.save_safetensors(tmp_path / "y.safetensors", {"b": tensors["b"]})
    (tmp_path / "model.safetensors.index.json").write_text(json.dumps({"weight_map": {"a": "x.safetensors", "b": "y.safetensors"}}))
    assert set(checkpoint.load_weights(tmp_path)) == {"a", "b"}
    (tmp_path / "bad.safetensors").write_bytes(b"\xff" * 16)
    with pytest.raises(ValueError):
        checkpoint.read_safetensors(tmp_path / "bad.safetensors")


def test_argument_structs_have_the_header_layout(tmp_path):
    names = {"spk_residual_norm_args": _lib.ResidualNormArgs, "spk_qk_prepare_args": _lib.QkPrepareArgs,
             "spk_sigmoid_attn_args": _lib.SigmoidAttnArgs, "spk_decay_attn_args": _lib.DecayAttnArgs,
             "spk_gated_norm_args": _lib.GatedNormArgs}
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


def test_components_cover_the_sources():
    listed = [n for group in build.COMPONENTS.values() for n in group]
    assert sorted(listed) == sorted(p.name for p in build.sources())
    some = {p.name for p in build.sources(("dense",))}
    assert "spk_capi.cu" in some and "spk_lif.cu" not in some
    assert build.library_path(("dense",)) != build.LIB_PATH


def test_host_argument_checks(lib):
    call = lambda name, args: getattr(lib, name)(ctypes.byref(args), None)
    assert lib.spk_residual_norm(None, None) == -4
    a = _lib.ResidualNormArgs(x=1, delta=1, w=1, out=1, n=4, width=0, dtype=_lib.F32)
    assert call("spk_residual_norm", a) == -2
    a.width, a.n = 8, 0
    assert call("spk_residual_norm", a) == 0
    a.n, a.mix, a.prev, a.positions, a.token_rows, a.token_edges, a.state_rows, a.x_out = 4, 1, 1, 1, 1, 1, 2, 1
    assert call("spk_residual_norm", a) == -6          # in place would race with the recomputed predecessor
    assert lib.spk_poly_norm(1, 1, 1e-5, 1, 2, 8, _lib.F16, None) == -1
    s = _lib.SigmoidAttnArgs(n=1, heads=3, kv_heads=2, dim=8, vdim=8, k_pad=8, v_pad=8, block_size=16, num_blocks=2, max_blocks=1)
    assert call("spk_sigmoid_attn", s) == -2           # heads not a multiple of kv_heads
    form = (_lib.BF16, 64, 64, 1, 1, 16)
    assert lib.spk_sigmoid_attn_tile_tokens(*form) == 128 and lib.spk_sigmoid_attn_tile_tokens(_lib.F32, 64, 64, 0, 0, 16) == 16
    assert lib.spk_sigmoid_attn_splits(*form, 64, 8, 2, 4096) == 4
    assert lib.spk_sigmoid_attn_splits(*form, 1, 8, 2, 512) == 2
    assert lib.spk_sigmoid_attn_splits(_lib.F32, 64, 64, 0, 0, 16, 1, 8, 2, 512) == 0
    d = _lib.DecayAttnArgs(n=1, heads=1, dim=4, vdim=4, state_rows=1, dtype=_lib.F32, q=1, k=1, v=1, state=1, decay_pow=1, out=1,
                           state_stride=8)
    assert call("spk_decay_attn_step", d) == -3        # rows of the state overlap
    d.state_stride = 16
    assert call("spk_decay_attn_chunks", d) == -2      # no chunk list
    assert lib.spk_decay_attn_workspace_bytes(3, 2, 8, 4) == 3 * 2 * 8 * 4 * 4
    assert lib.spk_meta_extend(0, 0, *([1] * 11), 4, 4, 0, 16, None, None) == -2


def test_portions_and_ledger():
    assert cut_portions([5, 3], None) == [[(0, 0, 5), (1, 0, 3)]]
    calls = cut_portions([5, 3, 9], 4)
    assert [sum(hi - lo for _, lo, hi in c) for c in calls] == [4, 4, 4, 4, 1]
    seen: dict[int, int] = {}
    for c in calls:
        assert len({i for i, _, _ in c}) == len(c)     # one portion per prompt and call
        for i, lo, hi in c:
            assert seen.get(i, 0) == lo
            seen[i] = hi
    assert seen == {0: 5, 1: 3, 2: 9}
    led = BlockLedger(4, 4, 3)
    assert led.extend_error([(0, 5)]) is None
    led.extend(0, 5)                                   # 2 blocks
    assert led.free == 2 and 0 in led.held
    led.advance()                                      # held rows sit out
    assert led.seq_lens[0] == 5 and led.blocks_next_step() == 0
    led.extend(0, 3)
    assert led.free == 2 and led.seq_lens[0] == 8
    led.held.discard(0)
    assert led.blocks_next_step() == 1
    led.advance()
    assert led.free == 1 and led.seq_lens[0] == 9
    assert "max_model_len" in led.extend_error([(0, 4)]) and "blocks" in led.extend_error([(1, 5)])
    assert led.extend_error([(1, 0)]) == "empty portion"
    led.release(0)
    assert led.free == 4 and not led.held


def test_prefill_plan_never_mixes_portions():
    plan = PrefillPlan([0, 5, 7], [5, 2, 40], [0, 31, 8], [3, 0, 1], torch.device("cpu"))
    tiles = plan.tiles(16).tolist()
    assert sorted(tiles) == sorted([[0, 5, 3, 0], [5, 2, 0, 31], [7, 16, 1, 8], [23, 16, 1, 24], [39, 8, 1, 40]])
    assert [t[3] for t in tiles] == sorted((t[3] for t in tiles), reverse=True)
    chunks, seqs = plan.chunks(16)
    assert seqs.tolist() == [[0, 1, 3, 0], [1, 1, 0, 31], [2, 3, 1, 8]]
    assert chunks.tolist() == [[0, 5, 0, 0], [5, 2, 1, 0], [7, 16, 2, 0], [23, 16, 2, 1], [39, 8, 2, 2]]


def test_tiled_pool_order_is_the_swizzle():
    pool = PagedKVPool(2, 3, 16, 100, torch.bfloat16, "cpu")
    assert pool.tiled and pool.pad == 128
    plain = torch.arange(2 * 16 * 3 * 100, dtype=torch.float32).view(32, 3, 100) % 251
    for b, h, r, d in ((0, 0, 0, 0), (0, 2, 5, 99), (1, 1, 15, 64), (1, 0, 9, 63)):
        at = (d // 64) * 16 * 64 + r * 64 + (((d // 8) % 8) ^ (r & 7)) * 8 + d % 8
        pool.data.view(2, 3, -1)[b, h, at] = plain[b * 16 + r, h, d].to(torch.bfloat16)
        assert pool.rows()[b * 16 + r, h, d] == plain[b * 16 + r, h, d]
    assert not PagedKVPool(2, 1, 16, 130, torch.bfloat16, "cpu").tiled and not PagedKVPool(2, 1, 8, 64, torch.bfloat16, "cpu").tiled
    assert not PagedKVPool(2, 1, 16, 64, torch.float32, "cpu").tiled


# ---- the plain implementation itself ---------------------------------------------------------------------------
def test_oracle_mechanisms_against_closed_forms():
    g = torch.Generator().manual_seed(1)
    rnd = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    # recurrence = decayed masked products
    q, k, v, decay = rnd(9, 2, 4), rnd(9, 2, 4), rnd(9, 2, 3), [0.7, 0.9]
    o, S = mo.decay_recurrence(q, k, v, decay)
    for h in range(2):
        i = torch.arange(9)
        m = torch.where(i[:, None] >= i[None, :], decay[h] ** (i[:, None] - i[None, :]).double(), torch.zeros((), dtype=torch.float64))
        assert torch.allclose(o[:, h], (q[:, h] @ k[:, h].T * m) @ v[:, h])
    o2, S1 = mo.decay_recurrence(q[:4], k[:4], v[:4], decay)
    o3, S2 = mo.decay_recurrence(q[4:], k[4:], v[4:], decay, S1)
    assert torch.allclose(torch.cat([o2, o3]), o) and torch.allclose(S2, S)
    # a rotated pair's product depends on the distance alone, and scaling divides the angle
    rot = dict(dims=6, base=100.0, scaling=dict(factor=3.0))
    a, b = rnd(1, 8), rnd(1, 8)
    dot = lambda p, s: (mo.rotate(a, p, rot) * mo.rotate(b, s, rot)).sum()
    assert torch.allclose(dot(17, 5), dot(29, 17))
    assert torch.allclose(mo.rotate(a, 6, rot), mo.rotate(a, 2, dict(dims=6, base=100.0)))
    assert torch.equal(mo.rotate(a, 9, rot)[:, 6:], a[:, 6:]) and torch.equal(mo.rotate(a, 9, None), a)
    # the last query sees every key, the first of the portion only those up to itself
    q, k, v = rnd(2, 4, 5), rnd(6, 2, 5), rnd(6, 2, 3)
    out = mo.sigmoid_attention(q, k, v, 0.3, rnd(4))
    assert out.shape == (2, 4, 3)
    k2 = k.clone()
    k2[5] += 1.0
    changed = (mo.sigmoid_attention(q, k2, v, 0.3, torch.zeros(4, dtype=torch.float64)) - mo.sigmoid_attention(q, k, v, 0.3, torch.zeros(4, dtype=torch.float64))).abs().amax((1, 2))
    assert changed[0] == 0 and changed[1] > 0
    x = rnd(3, 7)
    assert torch.allclose(mo.layer_norm(x, torch.ones(7, dtype=torch.float64), 1e-5), torch.nn.functional.layer_norm(x, (7,)))
    z = mo.poly_norm(x, torch.tensor([0.0, 0.0, 0.0, 2.5], dtype=torch.float64), 1e-5)
    assert (z == 2.5).all()
    s = mo.token_shift(x, torch.tensor([0.0, 1.0, 0.5, 0, 0, 0, 0], dtype=torch.float64))
    assert torch.equal(s[:, 0], x[:, 0]) and torch.equal(s[1:, 1], x[:-1, 1]) and s[0, 1] == 0 and torch.allclose(s[1:, 2], (x[1:, 2] + x[:-1, 2]) / 2)


def test_oracle_is_causal():
    cfg = mc.CONFIGS["mixed"]
    w = mo.as_float(mo.random_weights(cfg, 3))
    tokens = torch.randint(0, cfg["vocab"], (12,), generator=torch.Generator().manual_seed(4)).tolist()
    full = mo.forward(tokens, w, cfg)
    assert torch.allclose(mo.forward(tokens[:7], w, cfg), full[:7]) and full.shape == (12, cfg["vocab"])
    tokens[8] = (tokens[8] + 1) % cfg["vocab"]
    other = mo.forward(tokens, w, cfg)
    assert torch.allclose(other[:8], full[:8]) and (other[8:] - full[8:]).abs().amax(-1).min() > 1e-3
