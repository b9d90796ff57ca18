"""Nobodra: a decoder-only design whose sublayers read the residual stream ITSELF and whose norms sit on the sublayers'
outputs (`x <- x + norm1(mixer(x))`, `x <- x + norm2(ff(x))`, RMS norms with gains stored as their distance from one).
Two mixers:

* `delta`: a matrix state per head with ONE decay per head and token and a delta-rule write (`S <- g S;
  u = beta (v - S^T k); S <- S + k u^T; o = S^T q`); short convolutions with silu on q, k and v, unit-length q and k,
  the output RMS-normed per head and gated by silu of a full-rank projection.
* `attention`: grouped-query softmax attention over a sliding window whose values ARE the key projection (before norm
  and rotation; there is no value matrix), query and key heads RMS-normed, half-rotated pairs on part of each head.

Feed-forward (optional per layer): a mixture of experts without gates (`down(relu(up x)^2)`), the `top` largest biased
router logits chosen and weighted by the softmax over the chosen logits.

The model plugs into the same runtime as the package's other models: `setup_caches` builds every layer's cache or state
through `cache.get_cache_constructor` ("recent_global" = a ring of one window for attention, "state" = convolution tail
and matrix state for a delta layer), `forward(idx, input_pos, is_prefill)` is what `generation_utils.prefill` /
`decode_one_token` / `GraphedDecoder` call, and a step of any length continues from what the earlier steps left.  Matrix
products of prompt portions are cuBLAS (torch.mm, fp32 accumulation and output); one-token steps use this package's
product kernels; everything between products is a kernel of csrc/seq.  There is no CPU path.

Precision: weights, cache rows and product inputs are in the compute dtype (bf16 or fp32); the residual stream, norms,
convolutions, angles, attention scores and weights, router logits and weights, and everything of the recurrence are fp32
in both.

`OutputNorm` and `KeyValueAttention` take their sizes and constants as arguments so that another design can use them; the
delta rule is `tefovik.GatedDeltaRule` and the experts are `detatar.RoutedExperts`, both with other options.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

import torch
import torch.nn as nn
from torch import Tensor

from . import _lib, seq_ops
from .cache import get_cache_constructor
from .detatar import RoutedExperts, _out, _pad16, _padded_rows, _zeros
from .tefovik import GatedDeltaRule, _inv_freq, _product

MIXERS = ("delta", "attention")
FEED_FORWARDS = ("moe",)


# --------------------------------------------------------------------------------------------- configuration

@dataclass
class NobodraArgs:
    vocab_size: int
    dim: int
    layers: List[Dict[str, Any]]
    norm_eps: float
    block_size: int = 1 << 20      # angles are computed from the position: no table limits the length
    n_layer: int = field(init=False)

    def __post_init__(self):
        self.n_layer = len(self.layers)
        for i, layer in enumerate(self.layers):
            if layer.get("type") not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer type {layer.get('type')!r}")
            mlp = layer.get("mlp")
            if mlp and mlp.get("kind") not in FEED_FORWARDS:
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")

    @classmethod
    def from_config(cls, cfg: Dict[str, Any]):
        return cls(vocab_size=int(cfg["vocab"]), dim=int(cfg["width"]), layers=list(cfg["layers"]),
                   norm_eps=float(cfg["norm"]["eps"]))


# --------------------------------------------------------------------------------------------- mechanisms

class OutputNorm(nn.Module):
    """x + rms_norm(y) * (weight + gain_offset): the RMS norm of a sublayer's output and its sum into the stream in one
    pass, with the copy for the next product in the compute dtype.  y is a row per token or, as (rows, weights, slots),
    the weighted sum of the chosen experts' rows.  `then`: another OutputNorm-like gain (weight, eps) applied to the sum
    for that copy (the model's last norm)."""

    gain_offset = 1.0

    def __init__(self, dim: int, eps: float):
        super().__init__()
        self.eps = float(eps)
        self.weight = _zeros(dim, dtype=torch.float32)

    def forward(self, x: Tensor, result: Dict[str, Optional[Tensor]], x_act: Optional[Tensor] = None, x_out: Optional[Tensor] = None,
                then: Optional["OutputNorm"] = None):
        extra = {} if then is None else dict(next_w=then.weight, next_eps=then.eps, next_offset=then.gain_offset)
        seq_ops.post_norm(x, result["y"], self.weight, self.eps, self.gain_offset, wts=result.get("wts"), slot=result.get("slot"),
                          x_out=x_out, x_act=x_act, **extra)


class KeyValueAttention(nn.Module):
    """Grouped-query softmax attention with fp32 scores whose values are the projected keys themselves: a cached position
    holds the normed and rotated key beside the raw one.  Query and key heads are RMS-normed with a gain shared by the
    heads, the first `rot_dims` entries of each head turned by the position (pairs (i, i + rot_dims / 2)); query i sees key
    j <= i when `i - j < window` (window 0: every earlier key)."""

    def __init__(self, dim: int, heads: int, kv_heads: int, head_dim: int, scale: float, window: int, rot_base: float,
                 rot_dims: int, eps: float, dtype):
        super().__init__()
        if heads % kv_heads:
            raise ValueError("kv heads must divide the heads")
        if rot_dims % 2 or not 0 <= rot_dims <= head_dim:
            raise ValueError("rotary dims must be even and at most the head size")
        self.dim, self.heads, self.kv_heads, self.head_dim = dim, int(heads), int(kv_heads), int(head_dim)
        self.scale, self.window, self.rot_dims, self.eps = float(scale), int(window), int(rot_dims), float(eps)
        self.nq, self.nk = self.heads * self.head_dim, self.kv_heads * self.head_dim
        self.w_in = _zeros(_pad16(self.nq + self.nk), dim, dtype=dtype)      # rows: q | k | padding
        self.q_norm = _zeros(self.head_dim, dtype=torch.float32)
        self.k_norm = _zeros(self.head_dim, dtype=torch.float32)
        self.w_o = _zeros(dim, self.nq, dtype=dtype)
        self.register_buffer("inv_freq", _inv_freq(rot_base, self.rot_dims), persistent=False)

    def core(self, hp: Tensor, ip: Tensor, cache, one_token: bool) -> Tensor:
        """From the projection's fp32 rows to the input of the output projection [T, heads * head_dim]."""
        T, dev, dt = hp.shape[0], hp.device, self.w_o.dtype
        H, G, D = self.heads, self.kv_heads, self.head_dim
        q = torch.empty(T, H, D, dtype=torch.float32, device=dev)
        k = torch.empty(T, G, D, dtype=dt, device=dev)
        v = torch.empty(T, G, D, dtype=dt, device=dev)
        seq_ops.qkv_rope(hp, 0, self.nq, self.nq, H, G, D, D, self.q_norm, self.k_norm, self.eps, self.rot_dims, False,
                         self.inv_freq, None, ip, q, k, v)
        y = torch.empty(T, H, D, dtype=dt, device=dev)
        cache.sequence_step(q, k, v, ip, y, window=self.window, scale=self.scale)
        return y.view(T, self.nq)

    def input_conv(self, store):
        return None

    def close_one_token(self, hp: Tensor, ip: Tensor, cache, out: Tensor):
        """One token, from the input product's row to the mixer's output."""
        seq_ops.gemv_multi([(self.core(hp, ip, cache, True), self.w_o, out)])


class DeltaMixer(nn.Module):
    """`tefovik.GatedDeltaRule` as a mixer of its own: one decay per head, a full-rank output gate, and the projection
    that feeds it (rows q | k | v | b | a | g | padding)."""

    def __init__(self, dim: int, heads: int, kv_heads: int, head_dim: int, v_dim: int, taps: int, eps: float, dtype):
        super().__init__()
        self.rule = GatedDeltaRule(dim, heads, kv_heads, head_dim, v_dim, taps, None, None, eps, dtype, gate_act=_lib.ACT_SILU)
        self.w_in = _zeros(_pad16(self.rule.in_rows), dim, dtype=dtype)

    @property
    def w_o(self):
        return self.rule.w_o

    def core(self, hp: Tensor, ip: Tensor, state, one_token: bool) -> Tensor:
        return self.rule.core(hp, 0, ip, state, one_token)

    def input_conv(self, state):
        """One token: the short convolution runs inside the input product's launch (a channel is a row of it)."""
        return self.rule.conv.weight, state.vectors, self.rule.conv.act

    def close_one_token(self, hp: Tensor, ip: Tensor, state, out: Tensor):
        """One token, from the input product's row (its convolution applied) to the mixer's output: the recurrence, then the
        output product, which forms the normed and gated heads itself."""
        r = self.rule
        a = r.conv_width + r.heads
        g = a + r.a_rows
        o = r.scan(hp[:, :r.conv_width], hp[:, r.conv_width:a], hp[:, a:g], state)
        seq_ops.gemv_multi([(None, r.w_o, out)], pre=seq_ops.gated_heads_row(o, r.norm_w, hp[:, g:g + r.g_rows], r.gate_act, r.eps))


# --------------------------------------------------------------------------------------------- a layer

class NobodraBlock(nn.Module):
    """Mixer sublayer and optional feed-forward sublayer, each normed on its output."""

    def __init__(self, cfg: NobodraArgs, layer: Dict[str, Any], dtype):
        super().__init__()
        E, m, mlp = cfg.dim, layer["mixer"], layer.get("mlp")
        self.kind = layer["type"]
        if self.kind == "delta":
            self.mixer = DeltaMixer(E, int(m["heads"]), int(m.get("kv_heads", m["heads"])), int(m["dim"]), int(m["vdim"]), int(m.get("conv", 1)), cfg.norm_eps, dtype)
        else:
            rot = m.get("rot") or {}
            if int(m.get("vdim", m["dim"])) != int(m["dim"]):
                raise ValueError("values that are the projected keys are as wide as the keys")
            self.mixer = KeyValueAttention(E, int(m["heads"]), int(m.get("kv_heads", m["heads"])), int(m["dim"]), float(m["scale"]),
                                           int((m.get("mask") or {}).get("size", 0)), float(rot.get("base", 10000.0)),
                                           int(rot.get("dims", 0)), cfg.norm_eps, dtype)
        self.norm1 = OutputNorm(E, cfg.norm_eps)
        self.mlp = self.w_router = self.norm2 = None
        if mlp:
            r = mlp["router"]
            self.mlp = RoutedExperts(E, int(r["experts"]), 0, int(mlp["expert"]["ff"]), int(r["top"]), 1, 1, 0, _lib.ACT_RELU_SQ, dtype,
                                     scoring="softmax_chosen", gated=False)
            self.w_router = _zeros(_pad16(self.mlp.n_real), E, dtype=dtype)
            self.norm2 = OutputNorm(E, cfg.norm_eps)
        self.store = None           # the mixer's cache (attention) or recurrent state (delta)

    def mixed(self, x_act: Tensor, ip: Tensor, one_token: bool) -> Dict[str, Optional[Tensor]]:
        hp = _product(x_act, self.mixer.w_in, one_token)
        return dict(y=_product(self.mixer.core(hp, ip, self.store, one_token), self.mixer.w_o, one_token))

    def fed(self, x_act: Tensor, one_token: bool) -> Dict[str, Optional[Tensor]]:
        ids, wts = self.mlp.route(_product(x_act, self.w_router, one_token), 0)
        slot, y = self.mlp.expert_rows(ids, x_act)
        return dict(y=y, wts=wts, slot=slot)

    def forward(self, x: Tensor, x_act: Tensor, ip: Tensor, one_token: bool):
        """x fp32 [T, E] in place; x_act is its copy in the compute dtype (x itself in fp32)."""
        side = None if x_act is x else x_act
        self.norm1(x, self.mixed(x_act, ip, one_token), side)
        if self.mlp is not None:
            self.norm2(x, self.fed(x_act, one_token), side)

    def step_one_token(self, x: Tensor, copy: Optional[Tensor], ip: Tensor, pending: Optional[tuple]):
        """The same layer for one token; `copy` is scratch for the stream in the compute dtype (None in fp32).  `pending` is
        the sublayer result of the layer before with its norm: the input product's launch adds it to the stream (into a new
        buffer: its CTAs read the old row).  Then the mixer, the norm + sum + router in one launch, and the experts, whose
        weighted sum is this layer's pending result.  Returns (stream, pending)."""
        hp, mixed, conv = _out(self.mixer.w_in), _out(self.mixer.w_o), self.mixer.input_conv(self.store)
        if pending is None:
            seq_ops.gemv_multi([(x, self.mixer.w_in, hp)], conv=conv)
        else:
            result, norm = pending
            total = torch.empty_like(x)
            pre = seq_ops.output_norm_row(x, result["y"], norm.weight, norm.eps, norm.gain_offset, total, wts=result.get("wts"))
            seq_ops.gemv_multi([(None, self.mixer.w_in, hp)], pre=pre, conv=conv)
            x = total
        self.mixer.close_one_token(hp, ip, self.store, mixed)
        f = self.mlp
        if f is None:
            return x, (dict(y=mixed), self.norm1)
        if self.routes_with_norm():
            ids = torch.empty(1, f.top, dtype=torch.int32, device=x.device)
            wts = torch.empty(1, f.top, dtype=torch.float32, device=x.device)
            seq_ops.post_norm_route(x, mixed, self.norm1.weight, self.norm1.eps, self.norm1.gain_offset, self.w_router, f.correction,
                                    ids, wts, x_act=copy)
        else:
            self.norm1(x, dict(y=mixed), copy)
            ids, wts = f.route(_product(x if copy is None else copy, self.w_router, True), 0)
        _, y = f.expert_rows(ids, x if copy is None else copy)
        return x, (dict(y=y, wts=wts), self.norm2)

    # one CTA reads the whole router in the fused launch: beyond this a launch of its own, spread over the GPU, is faster
    ROUTER_BYTES = 1 << 19

    def routes_with_norm(self) -> bool:
        return self.w_router.numel() * self.w_router.element_size() <= self.ROUTER_BYTES

    def kernels_per_token(self):
        # input product (with the norm + sum of the layer before and the convolution), q/k/v rows + attention or the scan,
        # output product; norm + sum + router, experts up and down
        return (4 if self.kind == "attention" else 3) + (0 if self.mlp is None else 3 if self.routes_with_norm() else 5)


# --------------------------------------------------------------------------------------------- the model

class NobodraTransformer(nn.Module):
    """Same runtime surface as `model.Transformer`: setup_caches / reset_caches / forward / min_cache_length /
    get_cache_stats / prompt_cache_overflow, `config.block_size`, `config.n_layer`."""

    supports_prompt_portions = True

    def __init__(self, config: NobodraArgs, dtype=torch.bfloat16):
        super().__init__()
        assert dtype in (torch.bfloat16, torch.float32)
        self.config, self.dtype = config, dtype
        self.tok_embeddings = _zeros(config.vocab_size, config.dim, dtype=dtype)
        self.layers = nn.ModuleList(NobodraBlock(config, layer, dtype) for layer in config.layers)
        self.norm = OutputNorm(config.dim, config.norm_eps)
        self.output = _zeros(config.vocab_size, config.dim, dtype=dtype)
        self.max_batch_size = 1
        self.max_seq_length = 0
        # one-token steps through this package's product kernels; False = library products as in a prompt portion of
        # one token (used by A/B tests)
        self.fused_decode = True

    # ---- caches and state -------------------------------------------------------------------------
    def layer_cache_plan(self, cache_kwargs: Dict[str, Any], max_seq_length: int) -> Dict[str, Any]:
        """An attention layer keeps a ring of one window ("recent_global" without global tokens; "full" without a
        window), a delta layer a state of fixed size ("state": convolution tail and matrix state)."""
        ck = dict(cache_kwargs or {})
        ck["max_seq_length"] = max_seq_length
        strategies, lengths = [], []
        for layer in self.layers:
            window = layer.mixer.window if layer.kind == "attention" else None
            strategies.append("state" if window is None else ("recent_global" if window else "full"))
            lengths.append(0 if window is None else (window or max_seq_length))
        ck["cache_strategy"], ck["max_cache_length"] = strategies, lengths
        ck["global_tokens"] = 0
        ck["cache_bits"] = None
        ck["prompt_compression_strategy"] = ["none"] * len(self.layers)
        return ck

    def setup_caches(self, **kwargs):
        lengths = kwargs["max_cache_length"]
        for i, layer in enumerate(self.layers):
            ctor, _ = get_cache_constructor(kwargs["cache_strategy"][i])
            m = layer.mixer
            if layer.kind == "delta":
                layer.store = ctor(self.max_batch_size, **m.rule.state_spec())
            else:
                layer.store = ctor(self.max_batch_size, m.kv_heads, m.head_dim, self.dtype, max_cache_length=int(lengths[i]),
                                   max_seq_length=kwargs.get("max_seq_length"), global_tokens=0, cache_bits=None)
        self.max_seq_length = int(kwargs.get("max_seq_length") or max(lengths))

    def reset_caches(self):
        """Gives back what the finished sequence held: every slot empty, every state zero."""
        for layer in self.layers:
            layer.store.reset()

    def _unwindowed(self):
        return [l.kind == "attention" and not l.mixer.window for l in self.layers]

    def prompt_cache_overflow(self, prompt_length: int):
        return [u and prompt_length > l.store.max_cache_length for u, l in zip(self._unwindowed(), self.layers)]

    def min_cache_length(self):
        full = [l.store.max_cache_length for u, l in zip(self._unwindowed(), self.layers) if u]
        return min(full) if full else self.max_seq_length

    def get_cache_stats(self, prompt_len, gen_len):
        stats = {f"cache_slots_{i}": float(l.store.max_cache_length) for i, l in enumerate(self.layers)}
        stats["cache_memory_gb"] = sum(l.store.memory_usage() for l in self.layers)
        return stats

    # ---- one step: a whole prompt, a portion of it, or one token ----------------------------------
    @torch.no_grad()
    def forward(self, idx: Tensor, input_pos: Tensor, is_prefill: bool = True, mask: Optional[Tensor] = None,
                attn_top_k: Optional[float] = 1.0, logits_at: Optional[Tensor] = None,
                collect: Optional[list] = None) -> Tensor:
        """idx [1, T] token ids, input_pos [T] (or [1]) positions with input_pos[0] the first token's; returns fp32
        logits [1, n, vocab] for the rows `logits_at` (default: the last).  The step continues from the caches and
        state that earlier steps left.  `collect`, if a list, receives the residual stream after every layer."""
        assert attn_top_k in (None, 1, 1.0), "top-k attention is not part of this design"
        if any(l.store is None for l in self.layers):
            raise RuntimeError("Caches must be initialized first")
        tokens = idx.reshape(-1)
        if not tokens.is_cuda:
            raise _lib.CcError("this model runs on CUDA tensors only (no CPU fallback)")
        tokens = tokens if tokens.dtype == torch.int32 else tokens.to(torch.int32)
        ip = input_pos.reshape(-1)[:1]
        ip = ip if ip.dtype == torch.int32 else ip.to(torch.int32)
        T, E, dev, dt = tokens.numel(), self.config.dim, tokens.device, self.dtype
        one = T == 1 and self.fused_decode
        x = torch.empty(T, E, dtype=torch.float32, device=dev)
        x_act = x if dt == torch.float32 else torch.empty(T, E, dtype=dt, device=dev)
        seq_ops.embed_rows(tokens, self.tok_embeddings, x, 1.0)
        if one and collect is None and len(self.layers):
            return self._step_one_token(x, None if x_act is x else x_act, ip)
        if x_act is not x:
            seq_ops.gated_unit(x, 0, -1, x_act, _lib.ACT_NONE)
        for layer in self.layers:
            layer(x, x_act, ip, one)
            if collect is not None:
                collect.append(x.clone())
        rows = None if logits_at is None else logits_at.to(device=dev, dtype=torch.int64).contiguous()
        if rows is None:
            rows = torch.full((1,), T - 1, dtype=torch.int64, device=dev)
        xs_act = torch.empty(rows.numel(), E, dtype=dt, device=dev)
        seq_ops.sum_norm(self.norm.weight, self.norm.eps, x=x, center=False, gain_offset=self.norm.gain_offset, rows=rows, out_act=xs_act)
        return _product(xs_act, self.output, one).view(1, rows.numel(), -1)

    def _step_one_token(self, x: Tensor, copy: Optional[Tensor], ip: Tensor) -> Tensor:
        pending = None
        for layer in self.layers:
            x, pending = layer.step_one_token(x, copy, ip, pending)
        result, norm = pending
        xs_act = torch.empty_like(x) if copy is None else copy
        norm(x, result, xs_act, then=self.norm)
        logits = _out(self.output)
        seq_ops.gemv_multi([(xs_act, self.output, logits)])
        return logits.view(1, 1, -1)

    def kernels_per_token(self) -> int:
        """Launches of this package's kernels in one decode step (fused_decode)."""
        return 3 + sum(l.kernels_per_token() for l in self.layers)   # embedding row; last sum + both norms, head

    # ---- weights --------------------------------------------------------------------------------
    def load_tensors(self, tensors: Dict[str, Tensor]):
        """Fills the parameters from the checkpoint's tensor names ('embed', 'l<i>.norm1' / '.norm2', 'l<i>.mix.*',
        'l<i>.mlp.*', 'final.norm', 'head'), fusing the projection rows that read the same input."""
        used = set()

        def get(name, shape=None):
            if name not in tensors:
                raise KeyError(f"checkpoint has no tensor {name!r}")
            used.add(name)
            t = tensors[name]
            if shape is not None and tuple(t.shape) != tuple(shape):
                raise ValueError(f"{name}: shape {tuple(t.shape)} does not fit the configuration {tuple(shape)}")
            return t

        def put(param, value):
            param.data.copy_(value.to(param.dtype).reshape(param.shape))

        cfg = self.config
        E = cfg.dim
        put(self.tok_embeddings, get("embed", (cfg.vocab_size, E)))
        for i, b in enumerate(self.layers):
            p, q = f"l{i}.", f"l{i}.mix."
            put(b.norm1.weight, get(p + "norm1", (E,)).float())
            m = b.mixer
            if b.kind == "attention":
                put(m.w_in, _padded_rows([get(q + "q", (m.nq, E)), get(q + "k", (m.nk, E))], m.w_in.shape[0]))
                put(m.q_norm, get(q + "q.norm", (m.head_dim,)).float())
                put(m.k_norm, get(q + "k.norm", (m.head_dim,)).float())
                put(m.w_o, get(q + "o", (E, m.nq)))
            else:
                r = m.rule
                nk, nv, taps = r.kv_heads * r.head_dim, r.heads * r.v_dim, r.conv.taps
                put(m.w_in, _padded_rows([get(q + "q", (nk, E)), get(q + "k", (nk, E)), get(q + "v", (nv, E)), get(q + "b", (r.heads, E)),
                                          get(q + "a", (r.heads, E)), get(q + "g", (nv, E))], m.w_in.shape[0]))
                # a checkpoint may leave out the table of a one-tap convolution: that is the identity
                put(r.conv.weight, torch.cat([get(q + n + ".conv", (w, taps)).float() if taps > 1 or q + n + ".conv" in tensors else torch.ones(w, 1)
                                              for n, w in (("q", nk), ("k", nk), ("v", nv))]))
                put(r.A_log, get(q + "A_log", (r.heads,)).float())
                put(r.dt_bias, get(q + "dt_bias", (r.heads,)).float())
                put(r.norm_w, get(q + "norm", (r.v_dim,)).float())
                put(r.w_o, get(q + "o", (E, nv)))
            f = b.mlp
            if f is not None:
                q = p + "mlp."
                put(b.norm2.weight, get(p + "norm2", (E,)).float())
                put(b.w_router, _padded_rows([get(q + "router", (f.n_real, E))], b.w_router.shape[0]))
                put(f.correction, get(q + "router.b", (f.n_real,)).float())
                put(f.w_gu, torch.stack([get(f"{q}e{e}.up", (f.ff, E)) for e in range(f.n_real)]))
                put(f.w_d, torch.stack([get(f"{q}e{e}.down", (E, f.ff)) for e in range(f.n_real)]))
        put(self.norm.weight, get("final.norm", (E,)).float())
        put(self.output, get("head", (cfg.vocab_size, E)))
        return sorted(set(tensors) - used)

    @classmethod
    def from_config(cls, cfg: Dict[str, Any], dtype=torch.bfloat16):
        return cls(NobodraArgs.from_config(cfg), dtype)
