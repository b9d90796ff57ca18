"""CPU tests of the Nobodra design's host side: registry, configuration and shape errors, weight loading and fusing, the
cache plan, and the plain restatement's own invariants (the GPU tests hold the kernels to that restatement)."""
import json

import pytest
import torch

import nobodra_reference as R
from nobodra_utils import attention_layer, default_layers, delta_layer, make_config, moe, random_weights, reference_logits

F64 = torch.float64


def test_registry_builds_the_class_from_a_checkpoint_folder(tmp_path):
    from cold_compress_b200.checkpoint import load_checkpoint_folder, write_safetensors
    cfg = make_config(default_layers())
    W = random_weights(cfg, seed=1)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(tmp_path / "model.safetensors", W)
    model = load_checkpoint_folder(tmp_path, "cpu", torch.bfloat16)
    assert type(model).__name__ == "NobodraTransformer" and model.config.n_layer == 5 and model.supports_prompt_portions
    a = model.layers[0]                  # attention: fused q | k rows, zero padding, no value rows
    m = a.mixer
    assert m.w_in.shape == (96, 64) and torch.equal(m.w_in[:64], W["l0.mix.q"]) and torch.equal(m.w_in[64:96], W["l0.mix.k"])
    assert torch.equal(a.norm1.weight, W["l0.norm1"].float()) and a.norm1.gain_offset == 1.0
    f = a.mlp
    assert f.softmax_chosen and not f.gated and f.w_gu.shape == (6, 24, 64) and torch.equal(f.w_gu[4], W["l0.mlp.e4.up"])
    assert torch.equal(f.correction, W["l0.mlp.router.b"].float()) and torch.equal(f.w_d[2], W["l0.mlp.e2.down"])
    assert torch.equal(a.w_router[:6], W["l0.mlp.router"]) and a.w_router.shape == (16, 64) and float(a.w_router[6:].abs().sum()) == 0
    b = model.layers[1]                  # delta: q | k | v | b | a | g rows, one convolution table, no low-rank matrices
    r = b.mixer.rule
    assert r.w_a2 is None and r.w_g2 is None and r.dt_bias.numel() == 4
    at = 0
    for name, n in (("q", 32), ("k", 32), ("v", 48), ("b", 4), ("a", 4), ("g", 48)):
        assert torch.equal(b.mixer.w_in[at:at + n], W["l1.mix." + name]), name
        at += n
    assert at == r.in_rows and float(b.mixer.w_in[at:].abs().sum()) == 0
    assert torch.equal(r.conv.weight[32:64], W["l1.mix.k.conv"].float()) and torch.equal(r.conv.weight[64:], W["l1.mix.v.conv"].float())
    assert model.layers[2].mlp is None and model.layers[2].norm2 is None


def test_configuration_and_shape_errors():
    from cold_compress_b200.nobodra import NobodraArgs, NobodraTransformer
    cfg = make_config(default_layers())
    bad = json.loads(json.dumps(cfg))
    bad["layers"][1]["type"] = "wkv"
    with pytest.raises(ValueError, match="unknown mixer type"):
        NobodraArgs.from_config(bad)
    bad = json.loads(json.dumps(cfg))
    bad["layers"][0]["mlp"]["kind"] = "dense"
    with pytest.raises(ValueError, match="feed-forward"):
        NobodraArgs.from_config(bad)
    for layer, match in ((attention_layer(None, heads=5, kv_heads=2), "kv heads"), (delta_layer(None, heads=5, kv_heads=2), "kv heads"),
                         (attention_layer(None, dim=8, dims=10), "rotary"), (attention_layer(None, dims=5), "rotary"),
                         (attention_layer(moe(experts=3, top=4)), "choose 4 of 3")):
        with pytest.raises(ValueError, match=match):
            NobodraTransformer.from_config(make_config([layer]))
    bad = attention_layer(None)
    bad["mixer"]["vdim"] = 20
    with pytest.raises(ValueError, match="as wide as the keys"):
        NobodraTransformer.from_config(make_config([bad]))
    model = NobodraTransformer.from_config(cfg, torch.float32)
    W = random_weights(cfg, seed=2)
    short = dict(W)
    del short["l2.mix.v.conv"]
    with pytest.raises(KeyError, match="l2.mix.v.conv"):
        model.load_tensors(short)
    wrong = dict(W)
    wrong["l1.mix.dt_bias"] = wrong["l1.mix.dt_bias"][:2]
    with pytest.raises(ValueError, match="dt_bias"):
        model.load_tensors(wrong)
    extra = dict(W)
    extra["l9.unused"] = torch.zeros(1)
    assert model.load_tensors(extra) == ["l9.unused"]


def test_cache_plan_and_state_shapes():
    from cold_compress_b200.generation_utils import reset_caches, setup_caches
    from cold_compress_b200.nobodra import NobodraTransformer
    whole = attention_layer(None)
    del whole["mixer"]["mask"]
    model = NobodraTransformer.from_config(make_config([attention_layer(moe(), size=9), delta_layer(None, conv=3), whole]), torch.float32)
    ck = setup_caches(model, None, "cpu", 77, {})
    assert ck["cache_strategy"] == ["recent_global", "state", "full"] and ck["max_cache_length"] == [9, 0, 77]
    a, b, c = (l.store for l in model.layers)
    assert a.sequence_window() == 9 and a.sequence_kept() == 0 and c.sequence_window() == 0
    assert a.k_cache.shape == a.v_cache.shape == (1, 2, 9, 16) and c.k_cache.shape == (1, 2, 77, 16)
    assert b.vectors.shape == (2, 2 * 32 + 48) and b.matrix.shape == (4, 16, 12) and b.matrix.dtype == torch.float32
    assert model.min_cache_length() == 77 and model.prompt_cache_overflow(100) == [False, False, True]
    assert model.get_cache_stats(1, 1)["cache_slots_0"] == 9.0
    b.matrix.fill_(1.0)
    b.vectors.fill_(1.0)
    a.pos.fill_(3)
    reset_caches(model)
    assert float(b.matrix.abs().sum() + b.vectors.abs().sum()) == 0 and int(a.pos.max()) == -1


def test_there_is_no_cpu_path():
    from cold_compress_b200 import _lib
    from cold_compress_b200.generation_utils import setup_caches
    from cold_compress_b200.nobodra import NobodraTransformer
    model = NobodraTransformer.from_config(make_config(default_layers()), torch.float32)
    with pytest.raises(RuntimeError, match="initialized"):
        model(torch.zeros(1, 3, dtype=torch.int32), torch.arange(3))
    setup_caches(model, None, "cpu", 8, {})
    with pytest.raises(_lib.CcError, match="CUDA"):
        model(torch.zeros(1, 3, dtype=torch.int32), torch.arange(3))


# ----------------------------------------------------------------------------------------------- the restatement's own invariants

def test_restatement_is_causal():
    cfg = make_config(default_layers())
    W = random_weights(cfg, seed=3)
    tokens = torch.randint(0, cfg["vocab"], (40,), generator=torch.Generator().manual_seed(4)).tolist()
    full = reference_logits(cfg, W, tokens)
    assert (reference_logits(cfg, W, tokens[:25]) - full[:25]).abs().max() < 1e-9
    col = []
    reference_logits(cfg, W, tokens, col)
    assert len(col) == 5
    changed = list(tokens)
    changed[0] = (changed[0] + 1) % cfg["vocab"]         # the recurrence carries the first token past every window
    assert (reference_logits(cfg, W, changed)[39] - full[39]).abs().max() > 1e-7


def test_window_mask_reach():
    ok = R.window_mask(30, 5)
    assert ok[20, 16] and not ok[20, 15] and ok[20, 20] and not ok[20, 21] and int(ok[29].sum()) == 5
    assert bool((R.window_mask(30, 1) == torch.eye(30, dtype=torch.bool)).all()) and int(R.window_mask(30, 0)[29].sum()) == 30


def test_convolution_rotation_and_norms():
    g = torch.Generator().manual_seed(5)
    u, w = torch.randn(9, 4, generator=g, dtype=F64), torch.randn(4, 3, generator=g, dtype=F64)
    y = R.causal_conv(u, w)
    assert torch.allclose(y[0], u[0] * w[:, 2]) and torch.allclose(y[5], u[5] * w[:, 2] + u[4] * w[:, 1] + u[3] * w[:, 0])
    assert torch.allclose(R.causal_conv(u[:2], torch.randn(4, 5, generator=g, dtype=F64))[0].isfinite().double(), torch.ones(4, dtype=F64))
    x = torch.randn(5, 2, 8, generator=g, dtype=F64)
    r = R.rotate_halves(x, 100.0, 4)
    assert torch.allclose(r[0], x[0]) and torch.allclose(r[..., 4:], x[..., 4:])
    a = torch.tensor(3 * 100.0 ** -0.5, dtype=F64)       # position 3, second pair: entries 1 and 3
    assert torch.allclose(r[3, 1, 1], x[3, 1, 1] * torch.cos(a) - x[3, 1, 3] * torch.sin(a))
    assert torch.allclose(r[3, 1, 3], x[3, 1, 3] * torch.cos(a) + x[3, 1, 1] * torch.sin(a))
    assert torch.allclose((R.rms_around_one(u, torch.zeros(4, dtype=F64), 0.0) ** 2).mean(-1), torch.ones(9, dtype=F64))


def test_delta_rule_writes_overwrite_and_decays_forget():
    k = torch.zeros(3, 1, 4, dtype=F64)
    k[:, 0, 1] = 1.0
    v = torch.tensor([[[5.0]], [[7.0]], [[0.0]]], dtype=F64)
    one = torch.ones(3, 1, dtype=F64)
    o = R.delta_rule(k, k, v, torch.tensor([[1.0], [1.0], [0.0]], dtype=F64), one)
    assert o.flatten().tolist() == [5.0, 7.0, 7.0]        # a full write replaces what the key held; the read-out sees it
    o = R.delta_rule(k, k, v, torch.tensor([[1.0], [0.0], [0.0]], dtype=F64), 0.5 * one)
    assert o.flatten().tolist() == [5.0, 2.5, 1.25]
    assert torch.allclose(R.step_decay(torch.tensor([0.0], dtype=F64), torch.zeros(1, dtype=F64), torch.zeros(1, dtype=F64)), torch.tensor([0.5], dtype=F64))


def test_router_rules():
    ids, wts = R.route(torch.tensor([0.3, 2.0, -1.0, 1.5], dtype=F64), 2)
    assert ids.tolist() == [1, 3] and torch.allclose(wts, torch.softmax(torch.tensor([2.0, 1.5], dtype=F64), 0))
    ids, wts = R.route(torch.tensor([-90.0, -91.0], dtype=F64), 1)
    assert ids.tolist() == [0] and wts.tolist() == [1.0]
