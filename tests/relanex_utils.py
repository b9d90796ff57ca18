"""Small random Relanex checkpoints for the tests: configurations, weights under the checkpoint's tensor names, and
helpers to run the runtime.  The sizes here are the tests' own."""
from __future__ import annotations

import copy

import torch

from nevodra_utils import assert_rows_close, run_portions  # noqa: F401  (same drivers and bars for all designs)
from tidelorn_utils import row_error  # noqa: F401


def dense(ff=72):
    return {"kind": "dense", "ff": ff}


def attention_layer(mlp=None, heads=6, kv_heads=3, dim=16, vdim=20, base=800.0, dims=12, scale=None, scaling=(3.0, 100, 4.0, 0.5)):
    """scaling = (factor, original, fast, slow) or None."""
    rot = {"base": base, "dims": dims}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": rot,
                                                       "scale": scale or dim ** -0.5}}


def latent_layer(mlp=None, heads=3, dim=12, vdim=20, q_rank=28, kv_rank=24, size=13, scale=None):
    mixer = {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale or dim ** -0.5}
    if size:
        mixer["mask"] = {"size": size}
    return {"type": "latent_attention", "mlp": mlp, "mixer": mixer}


def mlstm_layer(mlp=None, heads=3, dim=12, vdim=20, gate_cap=7.0):
    return {"type": "mlstm", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap}}


def make_config(layers, width=64, vocab=131, eps=1e-5, mult=0.6, loop=None):
    cfg = {"architecture": "Relanex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "layers": copy.deepcopy(layers)}
    if loop:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg


def default_layers():
    """All three mixers, with and without a feed-forward."""
    return [latent_layer(dense(40)), mlstm_layer(dense()), attention_layer(None), mlstm_layer(None, heads=2, dim=20, vdim=8), latent_layer(None, size=9, heads=2),
            attention_layer(dense(48), heads=4, kv_heads=1, scaling=None)]


DEFAULT_LOOP = (1, 4, 3)     # layers 1, 2 and 3 run three times in a row


def random_weights(cfg, seed=0):
    """bf16 tensors under the checkpoint's names; every gain, offset and slope away from its neutral value; forget gates from
    fast to slow."""
    g = torch.Generator().manual_seed(seed)
    E, V = cfg["width"], cfg["vocab"]

    def rnd(*shape, s=1.0, mean=0.0):
        return (torch.randn(shape, generator=g) * s + mean).to(torch.bfloat16)

    W = {"embed": rnd(V, E), "head": rnd(V, E, s=E ** -0.5 * 3.0)}

    def norm(name, slope, offset=0.1):
        W[name], W[name + ".b"], W[name + ".alpha"] = rnd(E, s=0.3, mean=1.0), rnd(E, s=offset), rnd(s=0.1, mean=slope)

    norm("embed.norm", 0.8)
    norm("final.norm", 0.5)
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}."
        q = p + "mix."
        norm(p + "norm1", 0.6)
        norm(p + "norm1b", 0.9)
        H, D, Vd = m["heads"], m["dim"], m["vdim"]
        W[q + "o"] = rnd(E, H * Vd, s=(H * Vd) ** -0.5 * 1.5)
        if layer["type"] == "attention":
            G = m["kv_heads"]
            for n, w, s in (("q", H * D, 2.0), ("k", G * D, 2.0), ("v", G * Vd, 1.0)):
                W[q + n], W[q + n + ".b"] = rnd(w, E, s=E ** -0.5 * s), rnd(w, s=0.5)
            W[q + "sink"] = rnd(H, mean=0.5)
        elif layer["type"] == "latent_attention":
            R, C = m["q_rank"], m["kv_rank"]
            W[q + "dq"], W[q + "dkv"] = rnd(R, E, s=E ** -0.5), rnd(C, E, s=E ** -0.5)
            W[q + "dq.norm"], W[q + "dkv.norm"] = rnd(R, s=0.3, mean=1.5), rnd(C, s=0.3, mean=1.0)
            W[q + "uq"], W[q + "uk"], W[q + "uv"] = rnd(H * D, R, s=R ** -0.5), rnd(H * D, C, s=C ** -0.5 * 1.5), rnd(H * Vd, C, s=C ** -0.5)
        else:
            for n, w in (("q", H * D), ("k", H * D), ("v", H * Vd), ("g", H * Vd)):
                W[q + n] = rnd(w, E, s=E ** -0.5 * 1.5)
            W[q + "i"], W[q + "f"] = rnd(H, E, s=E ** -0.5 * 2.0), rnd(H, E, s=E ** -0.5 * 2.0)
            W[q + "i.b"], W[q + "f.b"] = rnd(H), rnd(H, s=2.0, mean=3.0)
            W[q + "norm"] = rnd(H * Vd, s=0.3, mean=1.0)
        mlp = layer.get("mlp")
        if mlp:
            F = mlp["ff"]
            norm(p + "norm2", 0.6)
            norm(p + "norm2b", 0.9)
            W[p + "mlp.gate"], W[p + "mlp.up"], W[p + "mlp.down"] = rnd(F, E, s=E ** -0.5 * 1.5), rnd(F, E, s=E ** -0.5 * 1.5), rnd(E, F, s=F ** -0.5 * 1.5)
    return W


def build_model(cfg, W, dtype, max_seq_length, device="cuda"):
    from cold_compress_b200.generation_utils import setup_caches
    from cold_compress_b200.relanex import RelanexTransformer
    model = RelanexTransformer.from_config(cfg, dtype)
    model.load_tensors(W)
    model = model.to(device).eval()
    setup_caches(model, None, device, max_seq_length, {})
    return model


def reference_logits(cfg, W, tokens, collect=None, dtype=torch.float64):
    import relanex_reference as R
    return R.forward(tokens, W, cfg, dtype=dtype, collect=collect)


def fp32_tolerance(cfg, W, tokens, want):
    """Three times the row error that fp32 rounding alone causes in the restatement itself (float32 against float64
    on the CPU): the bar for the fp32 kernels."""
    return max(3.0 * row_error(reference_logits(cfg, W, tokens, dtype=torch.float32), want).max().item(), 5e-6)
