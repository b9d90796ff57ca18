"""CPU tests of the Relanex design's host side: registry, configuration and shape errors, weight loading and fusing, layer
runs of a loop, the cache plan, stretched frequencies, and the plain restatement's own invariants (the GPU tests hold the
kernels to that restatement)."""
import json
import math

import pytest
import torch

import relanex_reference as R
from relanex_utils import DEFAULT_LOOP, attention_layer, default_layers, dense, latent_layer, make_config, mlstm_layer, random_weights, reference_logits

F64 = torch.float64


def test_registry_builds_the_class_from_a_checkpoint_folder(tmp_path):
    from cold_compress_b200.checkpoint import load_checkpoint_folder, write_safetensors
    cfg = make_config(default_layers(), loop=DEFAULT_LOOP)
    W = random_weights(cfg, seed=1)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(tmp_path / "model.safetensors", W)
    model = load_checkpoint_folder(tmp_path, "cpu", torch.bfloat16)
    assert type(model).__name__ == "RelanexTransformer" and model.config.n_layer == 12 and model.supports_prompt_portions
    assert [i for i, _ in model.config.runs()] == [0, 1, 2, 3, 1, 2, 3, 1, 2, 3, 4, 5]
    assert [i for i, l in enumerate(model.layers) if l.starts_pass] == [4, 7]
    assert model.layers[1].block is model.layers[4].block is model.layers[7].block and len(model.blocks()) == 6
    assert torch.equal(model.embed_norm.weight, W["embed.norm"].float()) and model.norm.alpha.item() == W["final.norm.alpha"].float().item()
    b = model.layers[0].block                 # latent: query latent rows | key/value latent rows, zero padding
    m = b.mixer
    assert m.w_in.shape[0] % 16 == 0 and torch.equal(m.w_in[:28], W["l0.mix.dq"]) and torch.equal(m.w_in[28:52], W["l0.mix.dkv"])
    assert float(m.w_in[52:].abs().sum()) == 0 and m.window == 13 and m.rot_dim == 0 and not m.gated and m.sink is None
    assert torch.equal(m.w_uk_t[1], W["l0.mix.uk"].view(3, 12, 24)[1].T) and torch.equal(b.w_gu[40:], W["l0.mlp.up"])
    b = model.layers[1].block                 # matrix memory: q | k | v | g | i | f rows
    m = b.mixer
    assert torch.equal(m.w_in[36:72], W["l1.mix.k"]) and torch.equal(m.w_in[132:192], W["l1.mix.g"]) and torch.equal(m.w_in[195:198], W["l1.mix.f"])
    assert m.gate_cap == 7.0 and torch.equal(m.f_bias, W["l1.mix.f.b"].float()) and m.norm_w.numel() == 60
    assert torch.equal(b.norm2b.bias, W["l1.norm2b.b"].float())
    b = model.layers[2].block                 # attention: biases in the same order as the rows
    m = b.mixer
    assert torch.equal(m.b_in[96:144], W["l2.mix.k.b"].float()) and torch.equal(m.sink, W["l2.mix.sink"].float()) and b.mlp is None
    assert model.layers[11].block.mixer.turn_gain == 1.0 and m.turn_gain != 1.0


def test_configuration_and_shape_errors():
    from cold_compress_b200.relanex import RelanexArgs, RelanexTransformer
    cfg = make_config(default_layers(), loop=DEFAULT_LOOP)

    def broken(change):
        bad = json.loads(json.dumps(cfg))
        change(bad)
        return bad

    with pytest.raises(ValueError, match="unknown mixer type"):
        RelanexArgs.from_config(broken(lambda c: c["layers"][1].update(type="conv")))
    with pytest.raises(ValueError, match="feed-forward"):
        RelanexArgs.from_config(broken(lambda c: c["layers"][0]["mlp"].update(kind="glu")))
    with pytest.raises(ValueError, match="loop"):
        RelanexArgs.from_config(broken(lambda c: c["loop"].update(stop=9)))
    with pytest.raises(ValueError, match="at least one layer"):
        RelanexArgs.from_config(broken(lambda c: (c["layers"].clear(), c.pop("loop"))))
    with pytest.raises(ValueError, match="kv heads"):
        RelanexTransformer.from_config(make_config([attention_layer(None, heads=5, kv_heads=2)]))
    with pytest.raises(ValueError, match="rotary"):
        RelanexTransformer.from_config(make_config([attention_layer(None, dims=18)]))
    with pytest.raises(ValueError, match="soft cap"):
        RelanexTransformer.from_config(make_config([mlstm_layer(None, gate_cap=0.0)]))
    model = RelanexTransformer.from_config(cfg, torch.float32)
    W = random_weights(cfg, seed=2)
    for name in ("l1.norm1b.alpha", "embed.norm.b", "l2.mix.v.b", "l1.mix.i.b"):
        with pytest.raises(KeyError, match=name):
            model.load_tensors({k: v for k, v in W.items() if k != name})
    with pytest.raises(ValueError, match="l0.mix.uq"):
        model.load_tensors(dict(W, **{"l0.mix.uq": W["l0.mix.uq"][:, :-1]}))
    with pytest.raises(ValueError, match="scalar"):
        model.load_tensors(dict(W, **{"final.norm.alpha": torch.zeros(2)}))
    assert model.load_tensors(dict(W, **{"l9.unused": torch.zeros(1)})) == ["l9.unused"]
    no_rank = broken(lambda c: c["layers"][0]["mixer"].pop("q_rank"))      # then the size is the tensor's shape
    model = RelanexTransformer.from_config(no_rank, torch.float32)
    assert model.load_tensors(W) == [] and model.layers[0].block.mixer.q_rank == 28


def test_cache_plan_and_state_shapes():
    from cold_compress_b200._lib import CcError
    from cold_compress_b200.generation_utils import reset_caches, setup_caches
    from cold_compress_b200.relanex import RelanexTransformer
    layers = [mlstm_layer(dense()), latent_layer(None, size=9), attention_layer(None), latent_layer(None, size=0)]
    model = RelanexTransformer.from_config(make_config(layers, loop=(0, 2, 2)), torch.float32)
    ck = setup_caches(model, None, "cpu", 77, {})
    assert ck["cache_strategy"] == ["state", "latent", "state", "latent", "full", "latent"]
    assert ck["max_cache_length"] == [0, 9, 0, 9, 77, 77]
    a, b, a2, b2, c, d = model.layers
    assert a.store is not a2.store and b.store is not b2.store and a.block is a2.block
    assert a.store.matrix.shape == (3, 12, 20) and a.store.vectors.shape == (3, 14)
    assert b.store.k_cache.shape == (1, 1, 9, 24) and b.store.v_cache.numel() == 0 and d.store.k_cache.shape == (1, 1, 77, 24)
    assert c.store.k_cache.shape == (1, 3, 77, 16) and c.store.v_cache.shape == (1, 3, 77, 20)
    assert model.min_cache_length() == 77 and model.prompt_cache_overflow(100) == [False, False, False, False, True, True]
    a.store.vectors.fill_(1.0)
    b.store.pos.fill_(3)
    reset_caches(model)
    assert float(a.store.vectors.abs().sum()) == 0 and int(b.store.pos.max()) == -1
    with pytest.raises(CcError):      # there is no CPU path
        model(torch.zeros(1, 3, dtype=torch.int32), torch.arange(3), True)
    short = RelanexTransformer.from_config(make_config([latent_layer(None, size=50), mlstm_layer(None)]), torch.float32)
    assert setup_caches(short, None, "cpu", 20, {})["max_cache_length"] == [50, 0] and short.min_cache_length() == 20


@pytest.mark.parametrize("base,dims,scaling", [(800.0, 12, (3.0, 100, 4.0, 0.5)), (10000.0, 64, (8.0, 4096, 32.0, 1.0)), (50.0, 2, (2.0, 9, 1.0, 1.0)),
                                                (1e6, 128, (1.0, 1000, 32.0, 1.0)), (500.0, 16, (4.0, 8, 64.0, 32.0))])
def test_stretched_frequencies(base, dims, scaling):
    from cold_compress_b200.tefovik import _stretched_inv_freq
    sc = dict(zip(("factor", "original", "fast", "slow"), scaling))
    f, gain = _stretched_inv_freq(base, dims, sc)
    want, amp = R.stretched_frequencies({"base": base, "dims": dims, "scaling": sc})
    assert f.dtype == torch.float32 and (f.double() / want - 1).abs().max() < 1e-7 and gain == pytest.approx(amp, abs=1e-12)
    plain, one = _stretched_inv_freq(base, dims, None)
    assert one == 1.0 and (plain.double() / R.stretched_frequencies({"base": base, "dims": dims})[0] - 1).abs().max() < 1e-7
    assert ((f <= plain * (1 + 1e-6)) & (f >= plain / sc["factor"] * (1 - 1e-6))).all()


# ----------------------------------------------------------------------------------------------- the restatement's own invariants

def test_restatement_is_causal_and_loops_add_the_embedding_output():
    cfg = make_config(default_layers(), loop=DEFAULT_LOOP)
    W = random_weights(cfg, seed=3)
    tokens = torch.randint(0, cfg["vocab"], (40,), generator=torch.Generator().manual_seed(4)).tolist()
    col = []
    full = reference_logits(cfg, W, tokens, col)
    assert len(col) == 12 and (reference_logits(cfg, W, tokens[:25]) - full[:25]).abs().max() < 1e-9
    assert R.layer_runs(cfg) == [(0, False), (1, False), (2, False), (3, False), (1, True), (2, False), (3, False), (1, True), (2, False),
                                 (3, False), (4, False), (5, False)]
    Wd = {k: v.double() for k, v in W.items()}
    first = R.bounded_norm(Wd["embed"][torch.tensor(tokens)], Wd, "embed.norm")
    assert torch.allclose(col[4], R.layer(col[3] + first, Wd, cfg, 1)) and torch.allclose(col[5], R.layer(col[4], Wd, cfg, 2))
    assert not torch.allclose(col[4], R.layer(col[3], Wd, cfg, 1))


def test_stabilised_memory_equals_the_plain_sum():
    """Without the maximum: S_t = sum_s exp(F_t - F_s + i_s) k_s v_s^T; the denominator is max(|n . q|, 1) on that scale."""
    g = torch.Generator().manual_seed(5)
    T, H, D, V = 20, 2, 5, 4
    q, k, v = (torch.randn(T, H, n, generator=g, dtype=F64) for n in (D, D, V))
    i, f = torch.randn(T, H, generator=g, dtype=F64) * 2, R.log_sigmoid(torch.randn(T, H, generator=g, dtype=F64) * 2)
    got = R.mlstm_cell(q, k, v, i, f)
    Fs = f.cumsum(0)
    for t in range(T):
        w = torch.exp(Fs[t] - Fs[:t + 1] + i[:t + 1])                                      # [s, H]
        dots = torch.einsum("shd,hd->sh", k[:t + 1], q[t]) * w
        want = torch.einsum("sh,shv->hv", dots, v[:t + 1]) / torch.maximum(dots.sum(0).abs(), torch.ones(H, dtype=F64))[:, None]
        assert torch.allclose(got[t], want, rtol=1e-4, atol=1e-7)      # up to the small constant in the denominator


def test_window_reach_sink_share_and_rotation():
    ok = R.visible(30, 5)
    assert ok[20, 16] and not ok[20, 15] and ok[20, 20] and not ok[20, 21] and int(ok[29].sum()) == 5 and int(R.visible(30)[29].sum()) == 30
    layer = attention_layer(None, heads=2, kv_heads=1)
    cfg = make_config([layer])
    W = {k: v.double() for k, v in random_weights(cfg, seed=6).items()}
    h = torch.randn(6, 64, generator=torch.Generator().manual_seed(7), dtype=F64)
    W["l0.mix.sink"] = torch.full((2,), -60.0, dtype=F64)      # weighs nothing: the first token's output is its own value
    free = R.attention(h, W, "l0.mix.", layer["mixer"], 1e-5)
    v0 = (h[0] @ W["l0.mix.v"].T + W["l0.mix.v.b"]).repeat(2) @ W["l0.mix.o"].T
    assert torch.allclose(free[0], v0)
    W["l0.mix.sink"] = torch.full((2,), 60.0, dtype=F64)       # takes everything
    assert R.attention(h, W, "l0.mix.", layer["mixer"], 1e-5).abs().max() < 1e-9
    rot = layer["mixer"]["rot"]
    x = torch.randn(5, 2, 16, generator=torch.Generator().manual_seed(8), dtype=F64)
    y = R.rotate(x, torch.arange(5), rot)
    f, amp = R.stretched_frequencies(rot)
    assert amp == pytest.approx(0.1 * math.log(3.0) + 1) and torch.allclose(y[..., 12:], x[..., 12:]) and torch.allclose(y[0, :, :12], amp * x[0, :, :12])
    assert torch.allclose(y[3, 1, 2], amp * (x[3, 1, 2] * torch.cos(3 * f[1]) - x[3, 1, 3] * torch.sin(3 * f[1])))
    s = torch.einsum("thd,shd->hts", R.rotate(x[:1].expand(5, 2, 16), torch.arange(5), rot), R.rotate(x[1:2].expand(5, 2, 16), torch.arange(5), rot))
    assert torch.allclose(s[:, 4, 3], s[:, 2, 1])              # scores depend on the distance
