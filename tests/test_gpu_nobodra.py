"""GPU tests of the Nobodra design: every mechanism's kernel against the plain restatement in nobodra_reference.py
(float64, CPU, whole sequences), then the model through the runtime: layer by layer, prompt against token-by-token
decoding, prompt portions down to two tokens, rows and states that are given back and used again, one key just inside
or just outside the window, an old write under slow decays, long decoding, other sizes, greedy generation through
generate() and the graph-captured decoder, and the trace replay command."""
import json

import pytest
import torch

import nobodra_reference as R
from nobodra_utils import (assert_rows_close, attention_layer, build_model, default_layers, delta_layer, fp32_tolerance, make_config,
                           moe, random_weights, reference_logits, row_error, run_portions)

pytestmark = pytest.mark.gpu
DEV = "cuda"
BF16_TOL = 6e-2
F64 = torch.float64


def _ops():
    from cold_compress_b200 import seq_ops
    return seq_ops


def _i32(*v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


def _tol(dtype, cfg, W, tokens, want):
    return BF16_TOL if dtype == torch.bfloat16 else fp32_tolerance(cfg, W, tokens, want)


def _close(got, want, rel):
    want = want.double()
    err = (got.detach().cpu().double() - want).abs().max().item()
    assert err <= rel * max(want.abs().max().item(), 1e-30), (err, want.abs().max().item())


# ----------------------------------------------------------------------------------------------- output norm

@pytest.mark.parametrize("E", [1, 50, 96, 640, 2052])
@pytest.mark.parametrize("T", [1, 70])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_output_norm_joins_the_stream(E, T, dtype):
    """x + norm(y) with a gain around one: in place and into a buffer of its own, y as a column range of wider rows, the
    copy for the next product, and the following norm."""
    ops = _ops()
    g = torch.Generator().manual_seed(E + T)
    x0, wide = torch.randn(T, E, generator=g) * 3, torch.randn(T, E + 5, generator=g) * 0.02      # eps matters
    w, w2 = torch.randn(E, generator=g) * 0.5, torch.randn(E, generator=g) * 0.5
    want = x0.double() + R.rms_around_one(wide[:, 3:3 + E].double(), w.double(), 1e-3)
    x, act = x0.to(DEV), torch.empty(T, E, device=DEV, dtype=dtype)
    ops.post_norm(x, wide.to(DEV)[:, 3:3 + E], w.to(DEV), 1e-3, 1.0, x_act=act)
    _close(x, want, 1e-6)
    assert torch.equal(act, x.to(dtype))
    x, out, act = x0.to(DEV), torch.empty(T, E, device=DEV), torch.empty(T, E, device=DEV, dtype=dtype)
    ops.post_norm(x, wide.to(DEV)[:, 3:3 + E].contiguous(), w.to(DEV), 1e-3, 1.0, x_out=out, x_act=act, next_w=w2.to(DEV), next_eps=1e-2, next_offset=1.0)
    assert torch.equal(x.cpu(), x0)
    _close(out, want, 1e-6)
    _close(act.float(), R.rms_around_one(want, w2.double(), 1e-2), 1e-5 if dtype == torch.float32 else 1e-2)


@pytest.mark.parametrize("T,E,top", [(1, 64, 3), (37, 64, 1), (5, 51, 4), (70, 256, 2)])
def test_output_norm_of_the_weighted_expert_rows(T, E, top):
    ops = _ops()
    g = torch.Generator().manual_seed(T)
    x0, rows = torch.randn(T, E, generator=g), torch.randn(T * top, E, generator=g)
    wts = torch.softmax(torch.randn(T, top, generator=g), -1)
    w = torch.randn(E, generator=g) * 0.5
    for slots in (None, torch.randperm(T * top, generator=g).to(torch.int32)):
        order = torch.arange(T * top) if slots is None else slots.long()
        mixed = (rows[order].double().view(T, top, E) * wts.double()[:, :, None]).sum(1)
        x = x0.to(DEV)
        ops.post_norm(x, rows.to(DEV), w.to(DEV), 1e-5, 1.0, wts=wts.to(DEV), slot=None if slots is None else slots.to(DEV))
        _close(x, x0.double() + R.rms_around_one(mixed, w.double(), 1e-5), 1e-6)


# ----------------------------------------------------------------------------------------------- one-token launches

@pytest.mark.parametrize("E,n,top", [(64, 6, 2), (51, 1, 1), (640, 40, 7), (2052, 9, 9), (4, 130, 3)])
@pytest.mark.parametrize("T", [1, 3])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_output_norm_with_the_router_that_reads_the_sum(E, n, top, T, dtype):
    ops = _ops()
    g = torch.Generator().manual_seed(E + n)
    x0, y, w = torch.randn(T, E, generator=g), torch.randn(T, E, generator=g), torch.randn(E, generator=g) * 0.5
    router, bias = (torch.randn(n + 3, E, generator=g) * E ** -0.5 * 0.1).to(dtype), torch.randperm(n, generator=g).float()
    want = x0.double() + R.rms_around_one(y.double(), w.double(), 1e-5)
    x, act = x0.to(DEV), torch.empty(T, E, device=DEV, dtype=dtype)
    ids, wts = torch.empty(T, top, dtype=torch.int32, device=DEV), torch.empty(T, top, device=DEV)
    ops.post_norm_route(x, y.to(DEV), w.to(DEV), 1e-5, 1.0, router.to(DEV), bias.to(DEV), ids, wts, x_act=act)
    _close(x, want, 1e-6)
    assert torch.equal(act, x.to(dtype))
    z = act.cpu().double() @ router[:n].double().T + bias.double()
    for t in range(T):
        wi, ww = R.route(z[t], top)
        assert ids[t].tolist() == wi.tolist()
        assert (wts[t].cpu().double() - ww).abs().max() < 1e-5


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("E,N,C,taps,top", [(64, 48, 40, 4, 0), (51, 9, 9, 2, 3), (640, 100, 33, 1, 2), (2052, 31, 0, 3, 4), (8, 1, 1, 7, 1)])
def test_products_that_form_the_normed_sum_and_convolve_their_rows(dtype, E, N, C, taps, top):
    """Several tokens one after another: the summed row is handed on, every row of the product sees it, and the first C
    rows pass a convolution whose tail moves on from call to call; a second product shares the row."""
    from cold_compress_b200 import _lib
    ops = _ops()
    g = torch.Generator().manual_seed(E)
    T = 9
    xs, ys = torch.randn(T, E, generator=g), torch.randn(T, max(top, 1), E, generator=g)
    wts = torch.softmax(torch.randn(T, max(top, 1), generator=g), -1)
    gain = torch.randn(E, generator=g) * 0.5
    W, W2 = (torch.randn(N, E, generator=g) * E ** -0.5).to(dtype), (torch.randn(5, E, generator=g) * E ** -0.5).to(dtype)
    table = torch.randn(C, taps, generator=g)
    mixed = (ys.double() * wts.double()[:, :, None]).sum(1) if top else ys[:, 0].double()
    stream = xs.double() + R.rms_around_one(mixed, gain.double(), 1e-4)
    rounded = stream.to(torch.float32).to(dtype).double()
    want = rounded @ W.double().T
    want2 = rounded @ W2.double().T
    if C:
        want = torch.cat([R.silu(R.causal_conv(want[:, :C], table.double())), want[:, C:]], 1)
    tail = torch.zeros(taps - 1, C, device=DEV)
    for t in range(T):
        out, out2, total = torch.empty(1, N, device=DEV), torch.empty(1, 5, device=DEV), torch.empty(1, E, device=DEV)
        pre = ops.output_norm_row(xs[t:t + 1].to(DEV), ys[t].to(DEV), gain.to(DEV), 1e-4, 1.0, total, wts=wts[t].to(DEV) if top else None)
        ops.gemv_multi([(None, W.to(DEV), out), (None, W2.to(DEV), out2)], pre=pre,
                       conv=(table.to(DEV), tail, _lib.ACT_SILU) if C else None)
        _close(total[0], stream[t], 1e-6)
        rel = 2e-5 if dtype == torch.float32 else 2e-2
        assert (out[0].cpu().double() - want[t]).abs().max() < rel * want.abs().max()
        assert (out2[0].cpu().double() - want2[t]).abs().max() < rel * want2.abs().max()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,V,N", [(4, 12, 48), (1, 1, 3), (9, 70, 20), (8, 128, 33)])
def test_product_of_normed_and_gated_heads(dtype, H, V, N):
    from cold_compress_b200 import _lib
    ops = _ops()
    g = torch.Generator().manual_seed(H * V)
    y, gate, w = torch.randn(1, H * V, generator=g) * 0.01, torch.randn(1, H * V + 4, generator=g) * 2, torch.randn(V, generator=g)
    W, out = (torch.randn(N, H * V, generator=g) * (H * V) ** -0.5).to(dtype), torch.empty(1, N, device=DEV)
    heads = R.rms_plain(y.double().view(H, V), w.double(), 1e-4) * R.silu(gate[:, 3:3 + H * V].double().view(H, V))
    ops.gemv_multi([(None, W.to(DEV), out)], pre=ops.gated_heads_row(y.to(DEV), w.to(DEV), gate.to(DEV)[:, 3:3 + H * V], _lib.ACT_SILU, 1e-4))
    _close(out[0], W.double() @ heads.reshape(-1), 1e-5 if dtype == torch.float32 else 2e-2)


def test_a_large_router_takes_a_launch_of_its_own():
    from cold_compress_b200.nobodra import NobodraBlock
    cfg = make_config(default_layers())
    W = random_weights(cfg, seed=15)
    tokens = torch.randint(0, cfg["vocab"], (30,), generator=torch.Generator().manual_seed(16)).tolist()
    want = reference_logits(cfg, W, tokens)
    model = build_model(cfg, W, torch.float32, 30)
    launches = model.kernels_per_token()
    keep, NobodraBlock.ROUTER_BYTES = NobodraBlock.ROUTER_BYTES, 0
    try:
        assert model.kernels_per_token() == launches + 2 * 3
        got = run_portions(model, tokens, (10,) + (1,) * 20)
    finally:
        NobodraBlock.ROUTER_BYTES = keep
    assert row_error(got, want).max() < fp32_tolerance(cfg, W, tokens, want)


def test_bad_arguments_are_errors_not_launches():
    from cold_compress_b200 import _lib
    ops = _ops()
    x = torch.zeros(1, 8, device=DEV)
    W, w = torch.zeros(4, 8, device=DEV), torch.zeros(8, device=DEV)
    with pytest.raises(AssertionError):
        ops.output_norm_row(x, x.clone(), w, 1e-5, 1.0, x)                      # other CTAs would read what one has written
    pre = ops.output_norm_row(x, x.clone(), w, 1e-5, 1.0, torch.zeros(1, 8, device=DEV))
    with pytest.raises(_lib.CcError, match="shared input row"):                 # the row is handed on by the first job's CTA
        ops.gemv_multi([(x, W, torch.zeros(1, 4, device=DEV)), (None, W, torch.zeros(1, 4, device=DEV))], pre=pre)
    with pytest.raises(_lib.CcError, match="post_norm_route"):
        ops.post_norm_route(x, x.clone(), w, 1e-5, 1.0, W, torch.zeros(2, device=DEV), torch.zeros(1, 3, dtype=torch.int32, device=DEV),
                            torch.zeros(1, 3, device=DEV))


# ----------------------------------------------------------------------------------------------- router and experts

@pytest.mark.parametrize("n,top", [(1, 1), (6, 2), (12, 12), (40, 5), (70, 1)])
def test_router_takes_the_largest_biased_logits_and_their_softmax(n, top):
    ops = _ops()
    g = torch.Generator().manual_seed(n)
    T = 64
    z, bias = torch.randn(T, n + 2, generator=g) * 3, torch.randn(n, generator=g)
    z[:8] += 200.0              # a softmax over the raw values would overflow or lose the losers' scale
    z[8:16] -= 200.0
    ids, wts = torch.empty(T, top, dtype=torch.int32, device=DEV), torch.empty(T, top, device=DEV)
    ops.moe_route(z.to(DEV)[:, 1:1 + n], bias.to(DEV), ids, wts, 1, 1, top, softmax_chosen=True)
    for t in range(T):
        biased = (z[t, 1:1 + n] + bias).double()          # the sum as the kernel forms it, in fp32
        wi, ww = R.route(biased, top)
        assert ids[t].tolist() == wi.tolist(), t
        assert (wts[t].cpu().double() - ww).abs().max() < 1e-6


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T", [1, 2, 4, 5, 33])
@pytest.mark.parametrize("n,top,ff,E", [(5, 2, 24, 48), (3, 3, 7, 50), (1, 1, 1, 2)])
def test_ungated_experts_few_tokens_and_grouped(dtype, T, n, top, ff, E):
    from cold_compress_b200 import _lib
    from cold_compress_b200.detatar import RoutedExperts
    g = torch.Generator().manual_seed(T * n)
    W = {"router": torch.randn(n, E, generator=g) * 0.2, "router.b": torch.randn(n, generator=g) * 2}
    for e in range(n):
        W[f"e{e}.up"], W[f"e{e}.down"] = torch.randn(ff, E, generator=g) * E ** -0.5, torch.randn(E, ff, generator=g)
    W = {k: v.to(dtype).float() for k, v in W.items()}
    h = torch.randn(T, E, generator=g).to(dtype).float()
    f = RoutedExperts(E, n, 0, ff, top, 1, 1, 0, _lib.ACT_RELU_SQ, dtype, scoring="softmax_chosen", gated=False)
    f.w_gu.data.copy_(torch.stack([W[f"e{e}.up"] for e in range(n)]))
    f.w_d.data.copy_(torch.stack([W[f"e{e}.down"] for e in range(n)]))
    f.correction.data.copy_(W["router.b"])
    f = f.to(DEV)
    z = (h @ W["router"].T).to(DEV)
    got = f(z, 0, None, h.to(DEV, dtype))
    want = R.mixture(h.double(), {k: v.double() for k, v in W.items()}, "", {"router": {"top": top}})
    _close(got, want, 1e-5 if dtype == torch.float32 else 2e-2)


# ----------------------------------------------------------------------------------------------- delta rule

def _delta_inputs(H, G, D, V, T, seed):
    g = torch.Generator().manual_seed(seed)
    q, k, v = torch.randn(T, G * D, generator=g), torch.randn(T, G * D, generator=g), torch.randn(T, H * V, generator=g)
    beta, a = torch.randn(T, H, generator=g), torch.randn(T, H, generator=g)
    return q, k, v, beta, a, torch.randn(H, generator=g) - 1.0, torch.randn(H, generator=g) * 0.7


def _delta_reference(q, k, v, beta, a, dt_bias, A_log, H, G, D, V):
    T = q.shape[0]
    d = lambda t: t.double()
    g = R.step_decay(d(a), d(A_log), d(dt_bias))
    return R.delta_rule(R.unit_vector(d(q).view(T, G, D)) * D ** -0.5, R.unit_vector(d(k).view(T, G, D)), d(v).view(T, H, V),
                        torch.sigmoid(d(beta)), g).reshape(T, H * V)


def _delta_run(q, k, v, beta, a, dt_bias, A_log, H, G, D, V, portions):
    """All inputs as column ranges of one wide row, as the model hands them over."""
    ops = _ops()
    row = torch.cat([q, k, v, beta, a], 1).to(DEV)
    state, out, at = torch.zeros(H, D, V, device=DEV), [], 0
    o1, o2, o3, o4 = G * D, 2 * G * D, 2 * G * D + H * V, 2 * G * D + H * V + H
    for n in portions:
        r = row[at:at + n]
        o = torch.empty(n, H * V, device=DEV)
        ops.delta_scan(r[:, :o1], r[:, o1:o2], r[:, o2:o3], r[:, o3:o4], r[:, o4:], dt_bias.to(DEV), A_log.to(DEV), state, o, H, G, D, V, D ** -0.5)
        out.append(o)
        at += n
    return torch.cat(out)


@pytest.mark.parametrize("H,G,D,V", [(1, 1, 1, 1), (4, 2, 16, 12), (6, 3, 40, 33), (2, 2, 64, 64), (3, 1, 128, 70), (2, 1, 130, 20),
                                     (1, 1, 256, 8), (40, 8, 12, 100)])
def test_delta_rule_with_one_decay_per_head(H, G, D, V):
    T = 150
    args = _delta_inputs(H, G, D, V, T, D + V)
    want = _delta_reference(*args, H, G, D, V)
    for portions in ((T,), (70, 80), (1,) * T, (2, 3, 64, 1, 1, 17, 62), (63, 65, 22)):
        _close(_delta_run(*args, H, G, D, V, portions), want, 1e-5)


@pytest.mark.parametrize("portions", [(700,), (5, 2, 300, 393), (9,) + (1,) * 691, (650,) + (1,) * 50], ids=["prompt", "portions", "decode", "decode_end"])
def test_an_old_write_is_read_back_under_slow_decay_and_lost_under_fast(portions):
    """A key that only position 7 writes (values 100 times the others', beta near one) is asked for at the last position:
    a head that decays slowly still returns it, a head that decays fast has lost it."""
    H, G, D, V, T = 2, 1, 24, 10, 700
    q, k, v, beta, a, dt_bias, A_log = _delta_inputs(H, G, D, V, T, 3)
    k[:, 0] = 0.0
    q[:, 0] = 0.0
    k[7], q[T - 1] = 0.0, 0.0
    k[7, 0] = q[T - 1, 0] = 5.0
    v[7], beta[7] = 100.0, 20.0
    a.zero_()
    dt_bias = torch.tensor([-9.0, 0.0])
    A_log = torch.zeros(2)
    want = _delta_reference(q, k, v, beta, a, dt_bias, A_log, H, G, D, V)
    assert want[-1, :V].abs().min() > 15 and want[-1, V:].abs().max() < 1e-12
    got = _delta_run(q, k, v, beta, a, dt_bias, A_log, H, G, D, V, portions)
    _close(got, want, 1e-5)
    assert (got[-1, :V].cpu().double() - want[-1, :V]).abs().max() < 1e-3


def _mixer_block(layer, W, width, dtype):
    from cold_compress_b200.nobodra import NobodraTransformer
    cfg = make_config([layer], width=width, vocab=7)
    model = NobodraTransformer.from_config(cfg, dtype)
    model.load_tensors(W)
    model = model.to(DEV).eval()
    from cold_compress_b200.generation_utils import setup_caches
    setup_caches(model, None, DEV, 400, {})
    return model.layers[0]


def _mixer_run(layer, h, portions, seed=5, dtype=torch.float32):
    """The mixer alone through the model's own block, beside the restatement of the same mixer."""
    width = h.shape[1]
    W = random_weights(make_config([layer], width=width, vocab=7), seed=seed)
    block = _mixer_block(layer, W, width, dtype)
    out, at = [], 0
    for n in portions:
        out.append(block.mixed(h[at:at + n].to(DEV, dtype).contiguous(), _i32(at), n == 1)["y"])
        at += n
    f = {"delta": R.delta, "attention": R.attention}[layer["type"]]
    want = f(h.to(dtype).double(), {k: v.double() for k, v in W.items()}, "l0.mix.", layer["mixer"], 1e-5)
    return torch.cat(out).cpu().double(), want


@pytest.mark.parametrize("kw", [dict(), dict(conv=1), dict(conv=7), dict(heads=1, kv_heads=1, dim=1, vdim=1, conv=2), dict(heads=6, kv_heads=1, dim=33, vdim=70)],
                         ids=["default", "one_tap", "seven_taps", "ones", "odd"])
def test_delta_mixer_carries_tail_and_state_across_portions(kw):
    h = torch.randn(90, 48, generator=torch.Generator().manual_seed(1))
    for portions in ((90,), (1,) * 90, (2, 5, 1, 1, 9, 2, 66, 4), (3,) * 30):
        got, want = _mixer_run(delta_layer(None, **kw), h, portions)
        _close(got, want, 2e-5)


# ----------------------------------------------------------------------------------------------- windowed attention

@pytest.mark.parametrize("kw", [dict(), dict(dims=16), dict(dims=0), dict(size=1), dict(heads=17, kv_heads=1, dim=8, dims=2, size=33), dict(heads=3, kv_heads=3, dim=70, dims=34, size=200),
                                dict(heads=1, kv_heads=1, dim=1, dims=0, size=5)],
                         ids=["default", "all_rotated", "unrotated", "window_1", "many_heads", "wide", "ones"])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_attention_mixer_in_portions_and_single_tokens(kw, dtype):
    h = torch.randn(150, 48, generator=torch.Generator().manual_seed(2))
    for portions in ((150,), (7, 2, 64, 33, 2, 40, 1, 1), (100,) + (1,) * 50, (1,) * 150):
        got, want = _mixer_run(attention_layer(None, **kw), h, portions, dtype=dtype)
        _close(got, want, 3e-5 if dtype == torch.float32 else 4e-2)


def test_values_are_the_projected_keys_before_norm_and_rotation():
    """With window 1 a query sees its own position only: the output is the raw key projection of its head's group."""
    layer = attention_layer(None, heads=4, kv_heads=2, dim=16, size=1)
    h = torch.randn(9, 48, generator=torch.Generator().manual_seed(3))
    W = {k: v.double() for k, v in random_weights(make_config([layer], width=48, vocab=7), seed=5).items()}
    raw = (h.double() @ W["l0.mix.k"].T).view(9, 2, 16).repeat_interleave(2, 1).reshape(9, 64) @ W["l0.mix.o"].T
    got, want = _mixer_run(layer, h, (4, 1, 1, 3))
    assert (want - raw).abs().max() < 1e-9
    _close(got, raw, 1e-5)


@pytest.mark.parametrize("mode", ["prompt", "portions", "decode"])
@pytest.mark.parametrize("where", ["oldest_in_window", "just_outside_window", "own_position", "position_0", "middle"])
def test_one_key_at_the_windows_edges_decides(mode, where):
    """One key's score stands far above the rest: inside the window it takes the whole softmax, one position outside it
    must not be seen."""
    from cold_compress_b200.cache import get_cache_constructor
    window, T, D = 44, 44 * 5 + 20, 16
    g = torch.Generator().manual_seed(3)
    q, k, v = torch.randn(T, 2, D, generator=g) * 0.1, torch.randn(T, 1, D, generator=g) * 0.1, torch.randn(T, 1, D, generator=g)
    last = T - 1
    j = {"oldest_in_window": last - window + 1, "just_outside_window": last - window, "own_position": last, "position_0": 0, "middle": last - window // 2}[where]
    k[j, 0], v[j] = 0.0, 100.0
    k[j, 0, 3] = 30.0
    q[last, :, 3] = 30.0
    want = R.softmax_attention(q.double(), k.double(), v.double(), 0.25, window)
    seen = where not in ("just_outside_window", "position_0")
    assert (want[last] - 100.0).abs().max() < 1e-6 if seen else want[last].abs().max() < 10
    cut = last - window
    portions = {"prompt": (T,), "portions": (3, 2, cut - 5, 2, T - cut - 2), "decode": (cut - 3,) + (1,) * (T - cut + 3)}[mode]
    ctor, _ = get_cache_constructor("recent_global")
    cache = ctor(1, 1, D, torch.float32, max_cache_length=window, max_seq_length=T, global_tokens=0, cache_bits=None).to(DEV)
    got, at = [], 0
    for n in portions:
        y = torch.empty(n, 2, D, device=DEV)
        cache.sequence_step(q[at:at + n].to(DEV), k[at:at + n].to(DEV), v[at:at + n].to(DEV), _i32(at), y, scale=0.25, window=window)
        got.append(y)
        at += n
    _close(torch.cat(got), want, 1e-5)


# ----------------------------------------------------------------------------------------------- the model in the runtime

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_layers_one_by_one_and_logits(dtype):
    cfg = make_config(default_layers())
    W = random_weights(cfg, seed=5, decisive=dtype == torch.bfloat16)
    tokens = torch.randint(0, cfg["vocab"], (41,), generator=torch.Generator().manual_seed(6)).tolist()
    ref_layers, got_layers = [], []
    want = reference_logits(cfg, W, tokens, ref_layers)
    model = build_model(cfg, W, dtype, 41)
    x = torch.tensor(tokens, dtype=torch.int32, device=DEV).view(1, -1)
    got = model(x, torch.arange(41, dtype=torch.int32, device=DEV), is_prefill=True, logits_at=torch.arange(41, device=DEV),
                collect=got_layers)[0]
    assert len(got_layers) == len(ref_layers) == 5 == model.config.n_layer
    for i, (a, b) in enumerate(zip(got_layers, ref_layers)):
        assert_rows_close((a.cpu().double() - b).abs().max(-1).values / b.abs().max(), dtype, 6e-2 if dtype == torch.bfloat16 else 2e-5, i)
    assert_rows_close(row_error(got, want), dtype, _tol(dtype, cfg, W, tokens, want))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_collecting_layers_of_a_single_token_changes_nothing(dtype):
    cfg = make_config(default_layers())
    W = random_weights(cfg, seed=7, decisive=True)
    model = build_model(cfg, W, dtype, 8)
    x, ip = _i32(5).view(1, 1), _i32(0)
    plain = model(x, ip, is_prefill=True).clone()
    model.reset_caches()
    col = []
    again = model(x, ip, is_prefill=True, collect=col)
    ref = []
    reference_logits(cfg, W, [5], ref)
    assert_rows_close(row_error(again[0], plain[0]), dtype, BF16_TOL if dtype == torch.bfloat16 else 1e-5)
    for a, b in zip(col, ref):
        _close(a, b, 5e-2 if dtype == torch.bfloat16 else 1e-5)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("portions", [(1,) * 70, (70,), (2,) * 35, (3, 11, 1, 1, 37, 2, 2, 12, 1), (8, 2, 3, 1, 56), (69, 1), (66, 4)],
                         ids=["token_by_token", "whole", "twos", "mixed", "around_window_edges", "last_alone", "long_then_short"])
def test_prompt_portions_and_decoding_agree_with_the_whole(dtype, portions):
    cfg = make_config(default_layers())
    W = random_weights(cfg, seed=9, decisive=dtype == torch.bfloat16)
    tokens = torch.randint(0, cfg["vocab"], (70,), generator=torch.Generator().manual_seed(10)).tolist()
    want = reference_logits(cfg, W, tokens)
    got = run_portions(build_model(cfg, W, dtype, 70), tokens, portions)
    assert_rows_close(row_error(got, want), dtype, _tol(dtype, cfg, W, tokens, want))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_one_token_kernels_equal_the_portion_kernels(dtype):
    """A decode step through the one-token product kernels against the same step through library products."""
    cfg = make_config(default_layers())
    W = random_weights(cfg, seed=15, decisive=dtype == torch.bfloat16)
    tokens = torch.randint(0, cfg["vocab"], (50,), generator=torch.Generator().manual_seed(16)).tolist()
    outs = []
    for fused in (True, False):
        model = build_model(cfg, W, dtype, 50)
        model.fused_decode = fused
        outs.append(run_portions(model, tokens, (30,) + (1,) * 20))
    assert_rows_close(row_error(outs[0], outs[1]), dtype, BF16_TOL if dtype == torch.bfloat16 else 1e-5)
    assert model.kernels_per_token() > 0


def test_sequences_one_after_another_reuse_states_and_rows():
    """Three sequences of unequal length through one model, rows and states given back in between: each equals itself
    alone."""
    from cold_compress_b200.generation_utils import reset_caches
    cfg = make_config(default_layers())
    W = random_weights(cfg, seed=11)
    g = torch.Generator().manual_seed(12)
    seqs = [torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for n in (45, 90, 13)]
    model = build_model(cfg, W, torch.float32, 90)
    for s, portions in zip(seqs, [(40, 1, 1, 1, 1, 1), (17, 60, 13), (13,)]):
        got = run_portions(model, s, portions)
        want = reference_logits(cfg, W, s)
        assert row_error(got, want).max() < fp32_tolerance(cfg, W, s, want)
        reset_caches(model)
        for l in model.layers:
            if l.kind == "delta":
                assert float(l.store.vectors.abs().sum() + l.store.matrix.abs().sum()) == 0
            else:
                assert int(l.store.cache_cts.item()) == 0 and int(l.store.pos.max()) == -1


def test_long_decoding_across_windows():
    """150 prompt tokens, then 330 tokens one by one: the rings wrap several times over decoded tokens and the states see
    every one of them."""
    cfg = make_config([attention_layer(moe(experts=4, top=2, ff=16), heads=2, kv_heads=1, dim=8, dims=4, size=50),
                       delta_layer(moe(experts=3, top=1, ff=16), heads=2, kv_heads=1, dim=8, vdim=8),
                       attention_layer(None, heads=2, kv_heads=2, dim=8, dims=8, size=140)], width=48, vocab=71)
    W = random_weights(cfg, seed=13)
    tokens = torch.randint(0, 71, (480,), generator=torch.Generator().manual_seed(14)).tolist()
    want = reference_logits(cfg, W, tokens)
    got = run_portions(build_model(cfg, W, torch.float32, 480), tokens, (150,) + (1,) * 330)
    assert row_error(got, want).max() < fp32_tolerance(cfg, W, tokens, want)


def _whole(layer):
    del layer["mixer"]["mask"]
    return layer


OTHER = [
    # every size that can be one is one
    ([attention_layer(moe(experts=1, top=1, ff=1), heads=1, kv_heads=1, dim=2, dims=2, size=1),
      delta_layer(moe(experts=1, top=1, ff=1), heads=1, kv_heads=1, dim=1, vdim=1, conv=1)], dict(width=4, vocab=5)),
    # 17 query heads on one key head, every expert chosen, long convolutions, no window
    ([delta_layer(moe(experts=5, top=5, ff=30), heads=17, kv_heads=1, dim=6, vdim=10, conv=6),
      _whole(attention_layer(moe(experts=10, top=4), heads=17, kv_heads=1, dim=8, dims=4)), attention_layer(None, heads=5, kv_heads=5, dim=6, dims=2, size=7)],
     dict(width=72, vocab=90)),
    # wide and odd sizes: heads beyond 64 and 128 columns, a window larger than the sequence, an odd width
    ([attention_layer(moe(experts=9, top=2, ff=10), heads=3, kv_heads=1, dim=66, dims=34, size=100, base=77.0),
      delta_layer(moe(experts=33, top=7, ff=9), heads=4, kv_heads=2, dim=70, vdim=37), delta_layer(None, heads=2, kv_heads=2, dim=140, vdim=6)],
     dict(width=69, vocab=61, eps=1e-3)),
    # only one kind of layer each, no feed-forward at all
    ([attention_layer(moe()), attention_layer(moe(experts=16, top=3))], dict(width=96, vocab=33)),
    ([delta_layer(moe()), delta_layer(moe(experts=16, top=3))], dict(width=96, vocab=33)),
    ([delta_layer(None), attention_layer(None)], dict(width=32, vocab=33)),
]


@pytest.mark.parametrize("layers,kw", OTHER, ids=["ones", "many_heads", "wide_odd", "attention_only", "delta_only", "no_feed_forward"])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_other_sizes(layers, kw, dtype):
    cfg = make_config(layers, **kw)
    W = random_weights(cfg, seed=21, decisive=dtype == torch.bfloat16)
    tokens = torch.randint(0, cfg["vocab"], (48,), generator=torch.Generator().manual_seed(22)).tolist()
    want = reference_logits(cfg, W, tokens)
    got = run_portions(build_model(cfg, W, dtype, 48), tokens, (5, 2, 30, 1, 1, 6, 1, 1, 1))
    assert_rows_close(row_error(got, want), dtype, _tol(dtype, cfg, W, tokens, want))


def test_checkpoint_folder_generate_and_graphed_decoder(tmp_path):
    """From a checkpoint folder through load_model, setup_caches and generate(): greedy tokens equal the restatement's
    arg-max continuation, with the prompt whole or in portions, eager or graph-captured."""
    from pathlib import Path
    from cold_compress_b200.checkpoint import write_safetensors
    from cold_compress_b200.generation_utils import compile_funcs, generate, load_model, reset_caches, setup_caches
    cfg = make_config(default_layers())
    W = random_weights(cfg, seed=17)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(tmp_path / "model.safetensors", W)
    prompt = torch.randint(0, cfg["vocab"], (33,), generator=torch.Generator().manual_seed(18)).tolist()
    new = 20
    seq, margins = list(prompt), []
    for _ in range(new):
        lg = reference_logits(cfg, W, seq)[-1]
        top = torch.topk(lg, 2).values
        margins.append((top[0] - top[1]).item())
        seq.append(int(lg.argmax()))
    model = load_model(Path(tmp_path), DEV, torch.float32, use_tp=False)
    assert type(model).__name__ == "NobodraTransformer"
    setup_caches(model, None, DEV, len(prompt) + new, {})
    for compile_, chunk in ((False, None), (False, 7), (True, 2)):
        prefill, decode = compile_funcs(compile_)
        out, _, stats = generate(model, torch.tensor(prompt, dtype=torch.int32, device=DEV), prefill, decode,
                                 max_new_tokens=new, prefill_chunk=chunk)
        out = out.tolist()
        assert out[:len(prompt)] == prompt and len(out) == len(seq)
        for i, (a, b) in enumerate(zip(out[len(prompt):], seq[len(prompt):])):
            assert a == b or margins[i] < 1e-3, (compile_, chunk, i)
            if a != b:
                break
        assert stats["decode_tokens"] == new
        reset_caches(model)


def test_trace_replay_command(tmp_path):
    """bin/trace_run as a user runs it: a checkpoint folder, steps on standard input (a whole prompt, portions with the
    last tokens alone, a second sequence after the first has ended), logits files and `done` lines."""
    import subprocess
    import sys
    from pathlib import Path
    import numpy as np
    from cold_compress_b200.checkpoint import write_safetensors
    root = Path(__file__).resolve().parent.parent
    cfg = make_config([delta_layer(moe()), attention_layer(moe(experts=9, top=3), size=32), attention_layer(None), delta_layer(None, conv=2)],
                      width=72, vocab=211)
    W = random_weights(cfg, seed=31, decisive=True)
    model_dir = tmp_path / "ckpt"
    model_dir.mkdir()
    (model_dir / "config.json").write_text(json.dumps(cfg))
    write_safetensors(model_dir / "model.safetensors", W)
    g = torch.Generator().manual_seed(32)
    a = torch.randint(0, 211, (75,), generator=g).tolist()
    b = torch.randint(0, 211, (41,), generator=g).tolist()
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[30:32], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[32:73], "want": [5, 40]}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": a[73:74], "want": [0]}], "end": []},
             {"step": 4, "entries": [{"id": "a", "tokens": a[74:75], "want": [0]}], "end": ["a"]},
             {"step": 5, "entries": [{"id": "b", "tokens": b, "want": [0, 20, 40]}], "end": ["b"]}]
    want = {0: [0, 29], 2: [37, 72], 3: [73], 4: [74]}
    la, lb = reference_logits(cfg, W, a), reference_logits(cfg, W, b)
    for dtype, tol in (("float32", 2e-4), ("bfloat16", 2 * BF16_TOL)):
        out = tmp_path / ("out_" + dtype)
        r = subprocess.run([sys.executable, str(root / "bin" / "trace_run"), "--model", str(model_dir), "--dtype", dtype,
                            "--out", str(out), "--max-tokens", "75"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                           capture_output=True, text=True, timeout=600)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == [f"done {i}" for i in range(6)]
        assert not (out / "1.f32").exists()
        for step, rows in want.items():
            got = torch.from_numpy(np.fromfile(out / f"{step}.f32", dtype="<f4").reshape(len(rows), -1).copy())
            assert row_error(got, la[rows]).max() < tol, (dtype, step)
        got = torch.from_numpy(np.fromfile(out / "5.f32", dtype="<f4").reshape(3, -1).copy())
        assert row_error(got, lb[[0, 20, 40]]).max() < tol
