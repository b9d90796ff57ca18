"""GPU tests of the Relanex design: every mechanism's kernel against the plain restatement in relanex_reference.py (float64,
CPU, whole sequences), then the model through the runtime: layer by layer, prompt against token-by-token decoding, prompt
portions down to two tokens, rows and states that are given back and used again, keys just inside and just outside the
window and far back, old writes of the matrix memory, long decoding, other sizes, greedy generation through generate() and
the graph-captured decoder, and the trace replay command."""
import json

import pytest
import torch

import relanex_reference as R
from relanex_utils import (DEFAULT_LOOP, assert_rows_close, attention_layer, build_model, default_layers, dense, fp32_tolerance, latent_layer,
                           make_config, mlstm_layer, random_weights, reference_logits, row_error, run_portions)

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


# ----------------------------------------------------------------------------------------------- bounded norms

def _norm(E, g, slope):
    W = {"n": torch.randn(E, generator=g), "n.b": torch.randn(E, generator=g), "n.alpha": torch.tensor([slope])}
    return {k: v.double() for k, v in W.items()}, tuple(W[k].to(DEV) for k in ("n.alpha", "n", "n.b"))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,E", [(1, 64), (1, 1), (5, 51), (300, 64), (7, 2052), (2, 130)])
def test_sum_with_bounded_norms_on_both_sides(dtype, T, E):
    ops = _ops()
    g = torch.Generator().manual_seed(T + E)
    W1, n1 = _norm(E, g, 0.7)
    W2, n2 = _norm(E, g, -1.3)
    x0, wide, first = torch.randn(T, E, generator=g) * 2, torch.randn(T, E + 4, generator=g) * 3, torch.randn(T, E, generator=g)
    y = wide[:, 4:]
    rel = 1e-6 if dtype == torch.float32 else 8e-3
    s1 = x0.double() + 0.35 * R.bounded_norm(y.double(), W1, "n")
    for add in (None, first):
        want = s1 if add is None else s1 + add.double()
        h, dev_add = torch.empty(T, E, dtype=dtype, device=DEV), None if add is None else add.to(DEV)
        x = x0.to(DEV)                                     # in place
        ops.bounded_sum(x, wide.to(DEV)[:, 4:], n1, 0.35, dev_add, x, n2, h)
        _close(x, want, 1e-6)
        _close(h.float(), R.bounded_norm(want, W2, "n"), rel)
        x, out = x0.to(DEV), torch.empty(T, E, device=DEV)      # into a buffer of its own
        ops.bounded_sum(x, wide.to(DEV)[:, 4:], n1, 0.35, dev_add, out, n2, h)
        assert torch.equal(x.cpu(), x0)
        _close(out, want, 1e-6)
        rows = torch.randperm(T, generator=g)[:max(1, T // 3)]
        hr = torch.empty(rows.numel(), E, dtype=dtype, device=DEV)
        ops.bounded_sum(x, wide.to(DEV)[:, 4:], n1, 0.35, dev_add, None, n2, hr, rows.to(DEV))
        assert torch.equal(hr, h[rows.to(DEV)])
    h = torch.empty(T, E, dtype=dtype, device=DEV)              # no sublayer result: the addition alone
    x = x0.to(DEV)
    ops.bounded_sum(x, add=first.to(DEV), x_out=x, next_norm=n2, h=h)
    _close(x, x0.double() + first.double(), 1e-6)
    _close(h.float(), R.bounded_norm(x0.double() + first.double(), W2, "n"), rel)


@pytest.mark.parametrize("table,act", [(torch.float32, torch.float32), (torch.bfloat16, torch.bfloat16), (torch.bfloat16, torch.float32)])
@pytest.mark.parametrize("T,E", [(1, 50), (9, 64), (200, 33)])
def test_embedding_rows_with_their_norms(table, act, T, E):
    ops = _ops()
    g = torch.Generator().manual_seed(E)
    W1, n1 = _norm(E, g, 0.9)
    W2, n2 = _norm(E, g, 0.4)
    embed, tokens = torch.randn(17, E, generator=g).to(table), torch.randint(0, 17, (T,), generator=g)
    x, h = torch.empty(T, E, device=DEV), torch.empty(T, E, dtype=act, device=DEV)
    ops.embed_bounded(tokens.to(DEV, torch.int32), embed.to(DEV), n1, x, n2, h)
    want = R.bounded_norm(embed.double()[tokens], W1, "n")
    _close(x, want, 1e-6)
    _close(h.float(), R.bounded_norm(want, W2, "n"), 1e-6 if act == torch.float32 else 8e-3)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("K,E", [(64, 48), (51, 33), (3, 1), (640, 200)])
@pytest.mark.parametrize("how", ["row", "gated_unit", "gated_heads"])
def test_product_whose_rows_join_the_stream(dtype, K, E, how):
    """A one-token product with the norm behind it, the sum and the next norm as its way out, for every way its input is
    formed; a second product rides along untouched."""
    from cold_compress_b200 import _lib
    ops = _ops()
    g = torch.Generator().manual_seed(K + E)
    W1, n1 = _norm(E, g, 0.8)
    W2, n2 = _norm(E, g, 0.5)
    W, V = (torch.randn(E, K, generator=g) * K ** -0.5).to(dtype), (torch.randn(5, K, generator=g) * K ** -0.5).to(dtype)
    x0, first = torch.randn(1, E, generator=g), torch.randn(1, E, generator=g)
    other, pre, job = torch.empty(1, 5, device=DEV), None, None
    if how == "row":
        inp = torch.randn(1, K, generator=g).to(dtype)
        row, job = inp.double()[0], (inp.to(DEV), W.to(DEV), None)
    elif how == "gated_unit":
        src = torch.randn(1, 2 * K + 3, generator=g)
        row = R.silu(src[0, 1:1 + K].double()) * src[0, 3 + K:].double()
        job = (src.to(DEV), W.to(DEV), None, _lib.ACT_SILU, 1, 3 + K)
    else:      # heads of K / parts entries, a gain over the whole row
        part = {64: 16, 51: 17, 3: 1, 640: 640}[K]
        y, gate, gain = torch.randn(1, K, generator=g) * 0.02, torch.randn(1, K, generator=g) * 2, torch.randn(K, generator=g)
        row = (R.rms_norm(y.double().view(-1, part), 1.0, 1e-4).reshape(-1) * gain.double()) * torch.sigmoid(gate.double()[0])
        pre, job = ops.gated_heads_row(y.to(DEV), gain.to(DEV), gate.to(DEV), _lib.ACT_SIGMOID, 1e-4, part=part), (None, W.to(DEV), None)
    want = W.double() @ row
    s = x0[0].double() + 0.3 * R.bounded_norm(want, W1, "n")
    rel = 1e-5 if dtype == torch.float32 else 2e-2
    for add, in_place in ((None, True), (first, False)):
        ws = s if add is None else s + add[0].double()
        x, h = x0.to(DEV), torch.empty(1, E, dtype=dtype, device=DEV)
        x_out = x if in_place else torch.empty(1, E, device=DEV)
        post = ops.bounded_way_out(x, n1, 0.3, x_out, n2, h, None if add is None else add.to(DEV))
        ops.gemv_multi([job, (job[0], V.to(DEV), other, *job[3:])], pre=pre, post=post)
        _close(x_out[0], ws, rel)
        _close(h[0].float(), R.bounded_norm(ws, W2, "n"), rel)
        _close(other[0], V.double() @ row, rel)
        assert in_place or torch.equal(x.cpu(), x0)


def test_bad_arguments_are_errors_not_launches():
    from cold_compress_b200 import _lib
    ops = _ops()
    x, z = torch.zeros(2, 8, device=DEV), torch.zeros(8, device=DEV)
    n = (torch.zeros(1, device=DEV), z, z)
    with pytest.raises(_lib.CcError, match="bounded_sum"):
        ops.bounded_sum(x)                                              # no output
    with pytest.raises(_lib.CcError, match="bounded_sum"):              # selected rows cannot go back into the stream
        ops.bounded_sum(x, x.clone(), n, 1.0, x_out=x, rows=torch.arange(2, device=DEV))
    with pytest.raises(AssertionError):
        ops.bounded_sum(x, x.clone(), (n[0], z[:4], z), 1.0, x_out=x)
    with pytest.raises(AssertionError):
        ops.gemv_multi([(x[:1], torch.zeros(4, 8, device=DEV), None)], post=ops.bounded_way_out(x[:1], n, 1.0, x[:1], n, x[1:]))
    state, aux, o = torch.zeros(1, 600, 4, device=DEV), torch.zeros(1, 602, device=DEV), torch.zeros(1, 4, device=DEV)
    row = torch.zeros(1, 1206, device=DEV)
    with pytest.raises(_lib.CcError, match="512"):
        ops.mlstm(row[:, :600], row[:, 600:1200], row[:, 1200:1204], row[:, 1204:1205], row[:, 1205:], z[:1], z[:1], 5.0, 1.0, state, aux, o,
                  1, 600, 4, path=_lib.MLSTM_SCAN)
    with pytest.raises(_lib.CcError, match="mlstm"):
        ops.mlstm(row[:, :600], row[:, 600:1200], row[:, 1200:1204], row[:, 1204:1205], row[:, 1205:], z[:1], z[:1], 0.0, 1.0, state, aux, o, 1, 600, 4)
    cache = _latent_cache(8, 10, torch.float32)
    with pytest.raises(_lib.CcError, match="looks back"):
        cache.latent_step(torch.zeros(1, 2, 8, device=DEV), torch.zeros(1, 1, 8, device=DEV), _i32(0), torch.zeros(1, 2, 8, device=DEV), 1.0, window=11)


# ----------------------------------------------------------------------------------------------- matrix memory

def _memory_inputs(H, D, V, T, seed, i_mean=0.0, f_mean=2.0):
    g = torch.Generator().manual_seed(seed)
    q, k, v = torch.randn(T, H * D, generator=g), torch.randn(T, H * D, generator=g), torch.randn(T, H * V, generator=g)
    i, f = torch.randn(T, H, generator=g) * 3, torch.randn(T, H, generator=g) * 3
    return q, k, v, i, f, torch.randn(H, generator=g) + i_mean, torch.randn(H, generator=g) * 2 + f_mean


def _memory_reference(args, H, D, V, cap, dtype=F64):
    q, k, v, i, f, ib, fb = (t.to(dtype) for t in args)
    T = q.shape[0]
    o = R.mlstm_cell(q.view(T, H, D) * D ** -0.5, k.view(T, H, D), v.view(T, H, V), cap * torch.tanh((i + ib) / cap),
                     R.log_sigmoid(cap * torch.tanh((f + fb) / cap)))
    return o.reshape(T, H * V)


def _memory_close(got, want, args, H, D, V, cap, rel=1e-5):
    """Within `rel` of the largest output plus three times the error of the fp32 restatement: a key sum that nearly cancels
    against the query makes an output that is large and ill-conditioned in any fp32 arithmetic."""
    own = (_memory_reference(args, H, D, V, cap, torch.float32).double() - want).abs().max()
    err = (got.detach().cpu().double() - want).abs().max()
    assert err <= rel * want.abs().max() + 3.0 * own, (err.item(), own.item(), want.abs().max().item())


def _memory_run(args, H, D, V, cap, portions, path=0, state=None):
    """All inputs as column ranges of one wide row, as the model hands them over."""
    ops = _ops()
    q, k, v, i, f, ib, fb = args
    row = torch.cat([q, k, v, i, f], 1).to(DEV)
    S, aux = state or (torch.zeros(H, D, V, device=DEV), torch.zeros(H, D + 2, device=DEV))
    a, b, c, d = H * D, 2 * H * D, 2 * H * D + H * V, 2 * H * D + H * V + H
    out, at = [], 0
    for n in portions:
        r = row[at:at + n]
        o = torch.full((n, H * V), float("nan"), device=DEV)
        ops.mlstm(r[:, :a], r[:, a:b], r[:, b:c], r[:, c:d], r[:, d:], ib.to(DEV), fb.to(DEV), cap, D ** -0.5, S, aux, o, H, D, V, path=path)
        assert int(aux[:, D + 1].view(torch.int32).abs().sum()) == 0          # the kernels' counter is back at zero
        out.append(o)
        at += n
    return torch.cat(out)


def _head_errors(got, want, H, V):
    """Error per (token, head), relative to that head's own output: a head's scale must not hide another's."""
    T = want.shape[0]
    d, w = (got.cpu().double() - want).view(T, H, V), want.view(T, H, V)
    return (d.pow(2).mean(-1) / (w.pow(2).mean(-1) + 1e-4 * w.pow(2).mean())).sqrt()


@pytest.mark.parametrize("H,D,V", [(1, 1, 1), (3, 12, 20), (2, 33, 70), (2, 64, 64), (1, 130, 36), (5, 8, 100), (1, 300, 7), (1, 520, 9)])
def test_memory_in_portions_by_scan_and_by_chunks(H, D, V):
    T, cap = 211, 6.0
    args = _memory_inputs(H, D, V, T, D + V)
    want = _memory_reference(args, H, D, V, cap)
    for path in (0, 1, 2):
        if path == 1 and D > 512:
            continue
        for portions in ((T,), (64, 64, 83), (65, 2, 63, 1, 80), (2, 3, 31, 32, 33, 1, 1, 108), (1,) * T):
            if path == 2 and len(portions) > 100:
                portions = (1,) * 9 + (T - 9,)
            got = _memory_run(args, H, D, V, cap, portions, path)
            assert _head_errors(got, want, H, V).max() < 3e-4, (path, portions[:4])
            _memory_close(got, want, args, H, D, V, cap)


@pytest.mark.parametrize("cap", [0.5, 15.0, 40.0])
@pytest.mark.parametrize("i_mean,f_mean", [(-30.0, 3.0), (30.0, 3.0), (0.0, -30.0), (0.0, 30.0)], ids=["closed_input", "open_input", "forget", "keep"])
def test_memory_with_saturated_gates(cap, i_mean, f_mean):
    """Gates at both ends of their soft cap: weights from e^-cap to e^cap, decays down to e^-cap and up to one."""
    H, D, V, T = 2, 16, 12, 300
    args = _memory_inputs(H, D, V, T, 3, i_mean, f_mean)
    want = _memory_reference(args, H, D, V, cap)
    for path, portions in ((1, (T,)), (2, (T,)), (0, (100, 2, 1, 1, 1, 150, 45))):
        got = _memory_run(args, H, D, V, cap, portions, path)
        assert torch.isfinite(got).all()
        _memory_close(got, want, args, H, D, V, cap)


@pytest.mark.parametrize("portions", [(900,), (5, 2, 300, 593), (9,) + (1,) * 891, (850,) + (1,) * 50], ids=["prompt", "portions", "decode", "decode_end"])
@pytest.mark.parametrize("path", [0, 2])
def test_an_old_write_is_read_back_where_the_gate_kept_it(portions, path):
    """A key that only position 7 writes is asked for at the last position: a head whose forget gate stays open returns its
    value, a head whose gate is half closed has lost it."""
    H, D, V, T = 2, 24, 10, 900
    if path == 2 and len(portions) > 100:      # single tokens are the scan's
        portions = (1, 1, 9, 64, 2, T - 77)
    q, k, v, i, f, ib, fb = _memory_inputs(H, D, V, T, 3)
    for h in range(H):
        k[:, h * D] = q[:, h * D] = 0.0
        k[7, h * D:(h + 1) * D] = q[T - 1, h * D:(h + 1) * D] = 0.0
        k[7, h * D] = q[T - 1, h * D] = 5.0
    v[7] = 100.0
    i.zero_(), f.zero_(), ib.zero_()
    args = (q, k, v, i, f, ib, torch.tensor([14.0, 0.0]))
    want = _memory_reference(args, H, D, V, 20.0)
    assert (want[-1, :V] - 100.0).abs().max() < 1 and want[-1, V:].abs().max() < 1e-9
    got = _memory_run(args, H, D, V, 20.0, portions, path)
    assert (got[-1].cpu().double() - want[-1]).abs().max() < 3e-2
    _memory_close(got, want, args, H, D, V, 20.0)


def test_running_maximum_starts_at_zero():
    """A first token with a closed input gate: the maximum stays at the start value plus the decay, so the denominator's floor
    is not one."""
    args = tuple(t[:3] for t in _memory_inputs(1, 4, 4, 3, 5)[:5]) + (torch.tensor([-8.0]), torch.tensor([6.0]))
    cap = 10.0
    want = _memory_reference(args, 1, 4, 4, cap)
    for path in (1, 2):
        S, aux = torch.zeros(1, 4, 4, device=DEV), torch.zeros(1, 6, device=DEV)
        _close(_memory_run(args, 1, 4, 4, cap, (3,), path, (S, aux)), want, 1e-5)
        i = cap * torch.tanh((args[3].double() + args[5].double()) / cap)
        f = R.log_sigmoid(cap * torch.tanh((args[4].double() + args[6].double()) / cap))
        m = torch.zeros(1, dtype=F64)
        for t in range(3):
            m = torch.maximum(f[t] + m, i[t])
        assert m.item() < 0 and abs(aux[0, 4].item() - m.item()) < 1e-6


# ----------------------------------------------------------------------------------------------- mixers through the model's block

def _mixer_run(layer, h, portions, seed=5, dtype=torch.float32, change=None, fused=True):
    """The mixer alone through the model's own block (projection, core, output product), beside the restatement."""
    from cold_compress_b200 import seq_ops
    cfg = make_config([layer], width=h.shape[1], vocab=7)
    W = random_weights(cfg, seed=seed)
    if change:
        change(W)
    model = build_model(cfg, W, dtype, h.shape[0])
    block, store = model.layers[0].block, model.layers[0].store
    m, out, at = block.mixer, [], 0
    for n in portions:
        one, x = n == 1 and fused, h[at:at + n].to(DEV, dtype).contiguous()
        if one:
            hp, y = torch.empty(1, m.w_in.shape[0], device=DEV), torch.empty(1, h.shape[1], device=DEV)
            seq_ops.gemv_multi([(x, m.w_in, hp)])
            inp, pre = m.core(hp, _i32(at), store, True)
            seq_ops.gemv_multi([(inp, m.w_o, y)], pre=pre)
        else:
            from cold_compress_b200.tidelorn import _mm
            inp, _ = m.core(_mm(x, m.w_in), _i32(at), store, False)
            y = _mm(inp, m.w_o)
        out.append(y)
        at += n
    want = R.MIXERS[layer["type"]](h.to(dtype).double(), {k: v.double() for k, v in W.items()}, "l0.mix.", layer["mixer"], 1e-5)
    return torch.cat(out).cpu().double(), want


PORTIONS = ((150,), (7, 2, 64, 33, 2, 40, 1, 1), (100,) + (1,) * 50, (1,) * 150)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("kw", [dict(), dict(heads=1, dim=1, vdim=1), dict(heads=5, dim=34, vdim=70, gate_cap=2.0)], ids=["default", "ones", "odd"])
def test_memory_mixer(kw, dtype):
    h = torch.randn(150, 48, generator=torch.Generator().manual_seed(1))
    for portions in PORTIONS:
        got, want = _mixer_run(mlstm_layer(None, **kw), h, portions, dtype=dtype)
        err = _head_errors(got, want, 1, 48)
        assert err.median() < (1e-5 if dtype == torch.float32 else 2e-2)
        _close(got, want, 5e-5 if dtype == torch.float32 else 6e-2)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("kw", [dict(), dict(scaling=None), dict(dims=16, scaling=(4.0, 30, 8.0, 1.0)), dict(dims=0, scaling=None), dict(heads=17, kv_heads=1, dim=8, dims=2, vdim=8),
                                dict(heads=3, kv_heads=3, dim=70, dims=34, vdim=35, scaling=(1.0, 50, 2.0, 2.0)), dict(heads=1, kv_heads=1, dim=2, dims=2, vdim=1)],
                         ids=["default", "unscaled", "all_rotated", "unrotated", "many_heads", "wide_factor_1", "small"])
def test_attention_mixer(kw, dtype):
    h = torch.randn(150, 48, generator=torch.Generator().manual_seed(2))
    for portions in PORTIONS:
        got, want = _mixer_run(attention_layer(None, **kw), h, portions, dtype=dtype)
        _close(got, want, 5e-5 if dtype == torch.float32 else 4e-2)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("kw", [dict(), dict(size=1), dict(size=0), dict(size=33, heads=17, dim=8, vdim=8, kv_rank=40), dict(size=149, dim=70, vdim=35, kv_rank=130, q_rank=9),
                                dict(size=200), dict(heads=1, dim=1, vdim=1, q_rank=1, kv_rank=1, size=5)],
                         ids=["default", "window_1", "no_window", "many_heads", "wide", "window_beyond", "ones"])
def test_latent_mixer(kw, dtype):
    h = torch.randn(150, 48, generator=torch.Generator().manual_seed(3))
    for portions in PORTIONS + ((14, 12, 2, 13, 13, 12, 14, 70),):
        got, want = _mixer_run(latent_layer(None, **kw), h, portions, dtype=dtype)
        _close(got, want, 5e-5 if dtype == torch.float32 else 4e-2)
        got, want = _mixer_run(latent_layer(None, **kw), h, portions, dtype=dtype, fused=False)      # expanded rows for single tokens too
        _close(got, want, 5e-5 if dtype == torch.float32 else 4e-2)


def test_a_larger_sink_takes_a_larger_share():
    h = torch.randn(40, 48, generator=torch.Generator().manual_seed(4))
    outs = []
    for sink in (-40.0, 1.0, 14.0):
        def change(W, sink=sink):
            W["l0.mix.sink"] = torch.full((6,), sink).to(torch.bfloat16)
        got, want = _mixer_run(attention_layer(None), h, (20,) + (1,) * 20, change=change)
        _close(got, want, 5e-5)
        outs.append(want.abs().sum())
    assert outs[0] > 1.02 * outs[1] and outs[1] > 1.5 * outs[2]


# ----------------------------------------------------------------------------------------------- decisive keys

def _latent_cache(width, slots, dtype):
    from cold_compress_b200.cache import get_cache_constructor
    ctor, _ = get_cache_constructor("latent")
    return ctor(1, 1, width, dtype, max_cache_length=slots, max_seq_length=slots, global_tokens=0, cache_bits=None).to(DEV)


@pytest.mark.parametrize("mode", ["prompt", "portions", "decode", "expanded_decode"])
@pytest.mark.parametrize("where", ["oldest_in_window", "just_outside_window", "own_position", "middle", "position_0"])
def test_one_latent_key_at_the_window_edges_decides(mode, where):
    """One position's latent scores far above the rest for the last query.  Inside the window it takes the whole softmax, one
    position outside it must not be seen."""
    size, T, E = 40, 40 * 4 + 17, 32
    layer = latent_layer(None, heads=2, dim=8, vdim=6, q_rank=E, kv_rank=E, size=size, scale=8.0)
    last = T - 1
    j = {"oldest_in_window": last - size + 1, "just_outside_window": last - size, "own_position": last, "middle": last - 19, "position_0": 0}[where]
    h = torch.randn(T, E, generator=torch.Generator().manual_seed(6)) * 0.5
    h[:, :2] = 0.0
    h[j, 0] = 12.0
    h[last, 1] = 12.0      # one input when j == last: both channels stand out

    def change(W):
        eye, q = torch.eye(E), "l0.mix."
        W[q + "dq"] = W[q + "dkv"] = eye.to(torch.bfloat16)
        uq, uk, uv = torch.zeros(16, E), torch.zeros(16, E), torch.randn(12, E, generator=torch.Generator().manual_seed(7)) * 0.1
        uq[::8, 1], uk[::8, 0] = 4.0, 4.0
        uv[:, 0] = 3.0
        for n, w in (("uq", uq), ("uk", uk), ("uv", uv)):
            W[q + n] = w.to(torch.bfloat16)

    cut = last - size
    portions = {"prompt": (T,), "portions": (3, 2, cut - 6, 2, T - cut - 1), "decode": (cut - 3,) + (1,) * (T - cut + 3),
                "expanded_decode": (cut - 3,) + (1,) * (T - cut + 3)}[mode]
    got, want = _mixer_run(layer, h, portions, change=change, fused=mode != "expanded_decode")
    plain, _ = _mixer_run(layer, torch.cat([h[:j] * 1.0, torch.zeros(1, E), h[j + 1:]]) if j != last else h, (T,), change=change)
    moved = (want[last] - plain[last]).abs().max()
    if where in ("just_outside_window", "position_0"):
        assert moved < 1e-6
    elif j != last:
        assert moved > 0.5
    _close(got, want, 5e-5)


@pytest.mark.parametrize("mode", ["prompt", "portions", "decode"])
def test_a_far_key_and_the_first_position_decide_in_the_global_attention(mode):
    T, E = 640, 40
    layer = attention_layer(None, heads=4, kv_heads=2, dim=16, vdim=12, dims=4, scale=1.0)
    for j in (0, 39, 511, 638):
        h = torch.randn(T, E, generator=torch.Generator().manual_seed(8)) * 0.3
        h[:, :2] = 0.0
        h[j, 0] = h[T - 1, 1] = 10.0

        def change(W):
            q = "l0.mix."
            for n in "qkv":
                W[q + n] = W[q + n] * 0.1
                W[q + n + ".b"] = W[q + n + ".b"] * 0.1
            W[q + "q"][9::16, 1] = 2.0          # an unrotated entry of every head
            W[q + "k"][9::16, 0] = 2.0
            W[q + "v"][:, 0] = 2.0

        portions = {"prompt": (T,), "portions": (33, 2, 500, 105), "decode": (600,) + (1,) * 40}[mode]
        got, want = _mixer_run(layer, h, portions, change=change)
        v = torch.zeros(1)
        base = _mixer_run(layer, torch.cat([h[:j], v.expand(1, E), h[j + 1:]]), (T,), change=change)[1]
        assert (want[T - 1] - base[T - 1]).abs().max() > 3
        _close(got, want, 5e-5)


def test_ring_rows_given_back_are_not_keys():
    """A second sequence after a longer one through the same latent ring: rows the first left behind must not be attended."""
    layer = latent_layer(None, size=20)
    cfg = make_config([layer], width=32, vocab=50)
    W = random_weights(cfg, seed=9)
    model = build_model(cfg, W, torch.float32, 70)
    g = torch.Generator().manual_seed(10)
    a, b = torch.randint(0, 50, (67,), generator=g).tolist(), torch.randint(0, 50, (31,), generator=g).tolist()
    run_portions(model, a, (30, 30, 7))
    store = model.layers[0].store
    assert sorted(store.pos[0, 0].tolist()) == list(range(47, 67)) and int(store.cache_cts.item()) == 20
    model.reset_caches()
    got, want = run_portions(model, b, (3, 1, 1, 19, 7)), reference_logits(cfg, W, b)
    assert row_error(got, want).max() < fp32_tolerance(cfg, W, b, want)
    assert sorted(store.pos[0, 0].tolist()) == list(range(11, 31))


# ----------------------------------------------------------------------------------------------- the model in the runtime

@pytest.mark.parametrize("T", [41, 1])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_layers_one_by_one_and_logits(dtype, T):
    cfg = make_config(default_layers(), loop=DEFAULT_LOOP)
    W = random_weights(cfg, seed=5)
    tokens = torch.randint(0, cfg["vocab"], (T,), generator=torch.Generator().manual_seed(6)).tolist()
    ref_layers, got_layers = [], []
    want = reference_logits(cfg, W, tokens, ref_layers)
    model = build_model(cfg, W, dtype, 41)
    x = torch.tensor(tokens, dtype=torch.int32, device=DEV).view(1, -1)
    got = model(x, torch.arange(T, dtype=torch.int32, device=DEV), is_prefill=True, logits_at=torch.arange(T, device=DEV),
                collect=got_layers)[0]
    assert len(got_layers) == len(ref_layers) == 12 == model.config.n_layer
    for i, (a, b) in enumerate(zip(got_layers, ref_layers)):
        assert_rows_close((a.cpu().double() - b).abs().max(-1).values / b.abs().max(), dtype, 6e-2 if dtype == torch.bfloat16 else 2e-5, i)
    assert_rows_close(row_error(got, want), dtype, _tol(dtype, cfg, W, tokens, want))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("portions", [(1,) * 90, (90,), (2,) * 45, (3, 11, 1, 1, 37, 2, 2, 12, 21), (8, 2, 3, 1, 76), (64, 26), (65, 25), (89, 1)],
                         ids=["token_by_token", "whole", "twos", "mixed", "around_window_edges", "chunk", "chunk_and_one", "last_alone"])
def test_prompt_portions_and_decoding_agree_with_the_whole(dtype, portions):
    cfg = make_config(default_layers(), loop=DEFAULT_LOOP)
    W = random_weights(cfg, seed=9)
    tokens = torch.randint(0, cfg["vocab"], (90,), generator=torch.Generator().manual_seed(10)).tolist()
    want = reference_logits(cfg, W, tokens)
    model = build_model(cfg, W, dtype, 90)
    got = run_portions(model, tokens, portions)
    assert_rows_close(row_error(got, want), dtype, _tol(dtype, cfg, W, tokens, want))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_one_token_kernels_equal_the_portion_kernels(dtype):
    """A decode step through the one-token product kernels against the same step through library products."""
    cfg = make_config(default_layers(), loop=DEFAULT_LOOP)
    W = random_weights(cfg, seed=15)
    tokens = torch.randint(0, cfg["vocab"], (50,), generator=torch.Generator().manual_seed(16)).tolist()
    outs = []
    for fused in (True, False):
        model = build_model(cfg, W, dtype, 50)
        model.fused_decode = fused
        outs.append(run_portions(model, tokens, (30,) + (1,) * 20))
    assert_rows_close(row_error(outs[0], outs[1]), dtype, BF16_TOL if dtype == torch.bfloat16 else 1e-5)


def test_launches_of_a_decode_step_are_as_many_as_claimed():
    """Every launch of a decode step is a kernel of this package: counted by the profiler on an eager step."""
    from torch.profiler import ProfilerActivity, profile
    from cold_compress_b200.generation_utils import model_step
    cfg = make_config(default_layers(), loop=DEFAULT_LOOP)
    model = build_model(cfg, random_weights(cfg, seed=19), torch.bfloat16, 40)
    run_portions(model, list(range(20)) , (18, 1, 1))
    x, ip = torch.tensor([[5]], dtype=torch.int32, device=DEV), _i32(20)
    with profile(activities=[ProfilerActivity.CUDA]) as p:
        model_step(model, x, ip, False)
        torch.cuda.synchronize()
    names = [e.name for e in p.events() if "kernel" in e.name and "Memcpy" not in e.name and "Memset" not in e.name]
    assert len(names) == model.kernels_per_token() and all("cc" in n for n in names), (len(names), model.kernels_per_token(), sorted(set(names)))


def test_sequences_one_after_another_reuse_rows_and_states():
    """Three sequences of unequal length through one model, caches and states given back in between: each equals itself
    alone."""
    from cold_compress_b200.generation_utils import reset_caches
    cfg = make_config(default_layers(), loop=DEFAULT_LOOP)
    W = random_weights(cfg, seed=11)
    g = torch.Generator().manual_seed(12)
    seqs = [torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for n in (45, 90, 13)]
    model = build_model(cfg, W, torch.float32, 90)
    for s, portions in zip(seqs, [(40, 1, 1, 1, 1, 1), (17, 60, 13), (13,)]):
        got, want = run_portions(model, s, portions), reference_logits(cfg, W, s)
        assert row_error(got, want).max() < fp32_tolerance(cfg, W, s, want)
        reset_caches(model)
        for l in model.layers:
            if l.block.kind == "mlstm":
                assert float(l.store.matrix.abs().sum()) == 0 and float(l.store.vectors.abs().sum()) == 0
            else:
                assert int(l.store.pos.max()) == -1 and int(l.store.cache_cts.item()) == 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_long_decoding_across_windows(dtype):
    """150 prompt tokens, then 330 tokens one by one: the rings wrap several times over decoded tokens."""
    cfg = make_config([latent_layer(dense(40), heads=2, dim=8, vdim=8, q_rank=12, kv_rank=16, size=50), mlstm_layer(None, heads=2, dim=8, vdim=8),
                       attention_layer(dense(24), heads=2, kv_heads=1, dim=8, vdim=4, dims=8), latent_layer(None, heads=1, dim=8, vdim=4, q_rank=8, kv_rank=8, size=140)],
                      width=48, vocab=71, loop=(0, 2, 2))
    W = random_weights(cfg, seed=13)
    tokens = torch.randint(0, 71, (480,), generator=torch.Generator().manual_seed(14)).tolist()
    want = reference_logits(cfg, W, tokens)
    model = build_model(cfg, W, dtype, 480)
    got = run_portions(model, tokens, (150,) + (1,) * 330)
    assert_rows_close(row_error(got, want), dtype, _tol(dtype, cfg, W, tokens, want))


OTHER = [
    # every size that can be one is one (rotary entries come in pairs)
    ([attention_layer(dense(1), heads=1, kv_heads=1, dim=2, vdim=1, dims=2), latent_layer(dense(1), heads=1, dim=1, vdim=1, q_rank=1, kv_rank=1, size=1),
      mlstm_layer(dense(1), heads=1, dim=1, vdim=1)], dict(width=2, vocab=3, mult=1.0)),
    # 17 query heads on one key head, a loop over the last layers, no feed-forward anywhere
    ([mlstm_layer(None, heads=5, dim=6, vdim=40, gate_cap=1.0), attention_layer(None, heads=17, kv_heads=1, dim=8, vdim=8, dims=6),
      latent_layer(None, heads=17, dim=8, vdim=6, q_rank=10, kv_rank=50, size=7)], dict(width=72, vocab=90, loop=(1, 3, 2))),
    # wide and odd sizes, a window longer than the sequence, four passes over one layer in the middle
    ([attention_layer(dense(30), heads=3, kv_heads=1, dim=66, vdim=34, dims=10, base=77.0), mlstm_layer(dense(14), heads=2, dim=130, vdim=70),
      latent_layer(dense(10), heads=5, dim=70, vdim=35, q_rank=33, kv_rank=130, size=100)], dict(width=70, vocab=60, loop=(1, 2, 4), mult=0.25, eps=1e-3)),
    # only one kind of layer each; a loop of one pass
    ([mlstm_layer(dense(64)), mlstm_layer(dense(20), heads=7, dim=4, vdim=4)], dict(width=96, vocab=33, loop=(0, 2, 1))),
    ([latent_layer(dense(64)), latent_layer(dense(8), size=3)], dict(width=96, vocab=33, loop=(0, 1, 4))),
    ([attention_layer(dense(64), scaling=None)], dict(width=96, vocab=33)),
]


@pytest.mark.parametrize("layers,kw", OTHER, ids=["ones", "many_heads", "wide_odd", "memory_only", "latent_only", "attention_only"])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_other_sizes(layers, kw, dtype):
    cfg = make_config(layers, **kw)
    W = random_weights(cfg, seed=21)
    tokens = torch.randint(0, cfg["vocab"], (48,), generator=torch.Generator().manual_seed(22)).tolist()
    want = reference_logits(cfg, W, tokens)
    model = build_model(cfg, W, dtype, 48)
    got = run_portions(model, tokens, (5, 2, 30, 1, 1, 6, 1, 1, 1))
    assert_rows_close(row_error(got, want), dtype, _tol(dtype, cfg, W, tokens, want))


def test_checkpoint_folder_generate_and_graphed_decoder(tmp_path):
    """From a checkpoint folder through load_model, setup_caches and generate(): greedy tokens equal the restatement's
    arg-max continuation, with the prompt whole or in portions, eager or graph-captured."""
    from pathlib import Path
    from cold_compress_b200.checkpoint import write_safetensors
    from cold_compress_b200.generation_utils import compile_funcs, generate, load_model, reset_caches, setup_caches
    cfg = make_config(default_layers(), loop=DEFAULT_LOOP)
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
    assert type(model).__name__ == "RelanexTransformer"
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
    cfg = make_config([mlstm_layer(dense(40)), latent_layer(dense(24), size=32), attention_layer(None)], width=72, vocab=211, loop=(1, 3, 2))
    W = random_weights(cfg, seed=31)
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
