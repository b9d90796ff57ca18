"""Small random Nobodra checkpoints for the tests: configurations, weights under the checkpoint's tensor names, and
helpers to run the runtime.  The sizes here are the tests' own."""
from __future__ import annotations

import copy

import torch

from nevodra_utils import assert_rows_close, run_portions  # noqa: F401  (same drivers and bars for all designs)
from tidelorn_utils import row_error  # noqa: F401


def moe(experts=6, top=2, ff=24):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def delta_layer(mlp=None, heads=4, kv_heads=2, dim=16, vdim=12, conv=4):
    return {"type": "delta", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def attention_layer(mlp=None, heads=4, kv_heads=2, dim=16, size=13, base=500.0, dims=8, scale=None):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "mask": {"size": size},
                      "rot": {"base": base, "dims": dims}, "scale": scale or dim ** -0.5}}


def make_config(layers, width=64, vocab=131, eps=1e-5):
    return {"architecture": "Nobodra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": copy.deepcopy(layers)}


def default_layers():
    """Both mixers, each with and without a feed-forward."""
    return [attention_layer(moe()), delta_layer(moe(experts=9, top=3, ff=20)), delta_layer(None, heads=3, kv_heads=3, dim=20, vdim=28, conv=2),
            attention_layer(None, heads=6, kv_heads=2, dim=12, size=9, dims=12), delta_layer(moe(experts=4, top=4), heads=6, kv_heads=2, vdim=8)]


def random_weights(cfg, seed=0, decisive=False):
    """bf16 tensors under the checkpoint's names; gains away from their neutral values, decays from fast to slow.
    `decisive` makes no choice of an expert a close call (small router weights, biases 1.5 apart): otherwise a few tokens
    sit where two logits differ by less than the bf16 error of the router's input, either choice is a correct bf16 result,
    and the tokens after such a one see it too.  The bf16 runs of the model use decisive weights and are held to a bar for
    every position; the fp32 runs route by the logits."""
    g = torch.Generator().manual_seed(seed)
    E, V = cfg["width"], cfg["vocab"]

    def rnd(*shape, s=1.0, mean=0.0):
        return (torch.randn(*shape, generator=g) * s + mean).to(torch.bfloat16)

    W = {"embed": rnd(V, E, s=1.0), "final.norm": rnd(E, s=0.2), "head": rnd(V, E, s=E ** -0.5 * 3.0)}
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}."
        q = p + "mix."
        W[p + "norm1"] = rnd(E, s=0.3, mean=-0.2)
        H, G, D = m["heads"], m["kv_heads"], m["dim"]
        if layer["type"] == "attention":
            W[q + "q"], W[q + "k"] = rnd(H * D, E, s=E ** -0.5), rnd(G * D, E, s=E ** -0.5)
            W[q + "q.norm"], W[q + "k.norm"] = rnd(D, s=0.3, mean=1.5), rnd(D, s=0.3, mean=1.5)
            W[q + "o"] = rnd(E, H * D, s=(H * D) ** -0.5)
        else:
            Vd, taps = m["vdim"], m["conv"]
            for n, w in (("q", G * D), ("k", G * D), ("v", H * Vd)):
                W[q + n], W[q + n + ".conv"] = rnd(w, E, s=E ** -0.5), rnd(w, taps, s=0.7)
            W[q + "b"], W[q + "a"] = rnd(H, E, s=E ** -0.5), rnd(H, E, s=E ** -0.5)
            W[q + "A_log"], W[q + "dt_bias"] = rnd(H, s=1.0, mean=-1.0), rnd(H, s=1.0, mean=-1.5)
            W[q + "norm"], W[q + "g"] = rnd(Vd, s=0.3, mean=1.0), rnd(H * Vd, E, s=E ** -0.5)
            W[q + "o"] = rnd(E, H * Vd, s=(H * Vd) ** -0.5)
        mlp = layer.get("mlp")
        if not mlp:
            continue
        W[p + "norm2"] = rnd(E, s=0.3, mean=-0.2)
        q = p + "mlp."
        n, F = mlp["router"]["experts"], mlp["expert"]["ff"]
        W[q + "router"] = rnd(n, E, s=E ** -0.5 * (0.05 if decisive else 1.0))
        W[q + "router.b"] = (1.5 * torch.randperm(n, generator=g)).to(torch.bfloat16) if decisive else rnd(n, s=0.7)
        for e in range(n):
            W[f"{q}e{e}.up"], W[f"{q}e{e}.down"] = rnd(F, E, s=E ** -0.5), rnd(E, F, s=F ** -0.5)
    return W


def build_model(cfg, W, dtype, max_seq_length, device="cuda"):
    from cold_compress_b200.generation_utils import setup_caches
    from cold_compress_b200.nobodra import NobodraTransformer
    model = NobodraTransformer.from_config(cfg, dtype)
    model.load_tensors(W)
    model = model.to(device).eval()
    setup_caches(model, None, device, max_seq_length, {})
    return model


def reference_logits(cfg, W, tokens, collect=None, dtype=torch.float64):
    import nobodra_reference as R
    return R.forward(tokens, W, cfg, dtype=dtype, collect=collect)


def fp32_tolerance(cfg, W, tokens, want):
    """Three times the row error that fp32 rounding alone causes in the restatement itself (float32 against float64
    on the CPU): the bar for the fp32 kernels."""
    return max(3.0 * row_error(reference_logits(cfg, W, tokens, dtype=torch.float32), want).max().item(), 5e-6)
