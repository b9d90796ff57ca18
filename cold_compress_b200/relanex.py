"""Relanex: a decoder-only design whose norms compute no statistics.  Every norm is element-wise and bounded,
`B(v) = w * tanh(alpha v) + b`, and sits in front of AND behind every sublayer: `x <- x + m * B1b(mixer(B1(x)))`, then
`x <- x + m * B2b(ff(B2(x)))`, with one constant m for the model; the embedding rows and the model's end have one each.
Three mixers:

* `attention`: grouped-query causal softmax attention with biases on q, k and v, interleaved rotary pairs whose
  frequencies are stretched for a longer context, and a learned sink logit per head in the softmax denominator.
* `latent_attention`: keys and values are up-projections of one RMS-normed latent per position, queries go through a latent
  of their own; no positions; a sliding window.
* `mlstm`: a matrix memory per head with exponential gates, stabilised by a running maximum
  (`S <- exp(f + m - m') S + exp(i - m') k v^T`, a key sum n likewise, `o = S^T q / max(|n . q|, exp(-m'))`); head outputs
  RMS-normed and gated by a sigmoid.

Feed-forward (optional per layer): `down(silu(gate x) * up x)`.  A run of consecutive layers can be repeated with the same
weights: every pass has caches and state of its own, and every pass but the first starts by adding the embedding output.

The model plugs into the same runtime as the package's other models: `setup_caches` builds every layer run's cache or state
through `cache.get_cache_constructor` ("full" rows for attention, "latent" rows in a ring of one window, "state" for the
matrix memory), `forward(idx, input_pos, is_prefill)` is what `generation_utils.prefill` / `decode_one_token` /
`GraphedDecoder` call, and a step of any length continues from what the earlier steps left.  Since a bounded norm needs one
channel only, the norm behind a sublayer, the residual sum and the next sublayer's norm are the way out of the sublayer's
last product: a row of that product per channel in a one-token step, one element-wise launch after the library product in a
prompt portion.  Matrix products of prompt portions are cuBLAS (torch.mm, fp32 accumulation and output); one-token steps
use this package's product kernels; everything between products is a kernel of csrc/seq.  There is no CPU path.

Precision: weights, cache rows and product inputs are in the compute dtype (bf16 or fp32); the residual stream, norms,
angles, attention scores and weights and everything of the recurrence are fp32 in both.

`BoundedNorm`, `BiasedRotaryAttention` and `MatrixMemory` take their sizes and constants as arguments so that another
design can use them; the latent attention and the feed-forward are the ones of `detatar` with other options.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

import torch
import torch.nn as nn
from torch import Tensor

from . import _lib, seq_ops
from .cache import get_cache_constructor
from .detatar import GatedMLP, LatentAttention, _out, _pad16, _padded_rows, _zeros
from .nevodra import loop_runs
from .tefovik import _product, _stretched_inv_freq
from .tidelorn import _mm

MIXERS = ("attention", "latent_attention", "mlstm")
FEED_FORWARDS = ("dense",)


# --------------------------------------------------------------------------------------------- configuration

@dataclass
class RelanexArgs:
    vocab_size: int
    dim: int
    layers: List[Dict[str, Any]]
    norm_eps: float
    residual_mult: float
    loop_start: int = 0
    loop_stop: int = 0
    loop_times: int = 1
    block_size: int = 1 << 20      # angles are computed from the position: no table limits the length
    n_layer: int = field(init=False)

    def __post_init__(self):
        if not self.layers:
            raise ValueError("a model needs at least one layer")
        if not (0 <= self.loop_start <= self.loop_stop <= len(self.layers)) or self.loop_times < 1:
            raise ValueError("loop: start <= stop must lie within the layers and times must be positive")
        for i, layer in enumerate(self.layers):
            if layer.get("type") not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer type {layer.get('type')!r}")
            mlp = layer.get("mlp")
            if mlp and mlp.get("kind") not in FEED_FORWARDS:
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
        self.n_layer = len(self.runs())

    def runs(self):
        """[(layer index, pass number or None)] in running order."""
        return loop_runs(len(self.layers), self.loop_start, self.loop_stop, self.loop_times)

    @classmethod
    def from_config(cls, cfg: Dict[str, Any]):
        loop = cfg.get("loop") or {}
        return cls(vocab_size=int(cfg["vocab"]), dim=int(cfg["width"]), layers=list(cfg["layers"]), norm_eps=float(cfg["norm"]["eps"]),
                   residual_mult=float(cfg.get("residual_mult", 1.0)), loop_start=int(loop.get("start", 0)),
                   loop_stop=int(loop.get("stop", 0)), loop_times=int(loop.get("times", 1)))


# --------------------------------------------------------------------------------------------- mechanisms

class BoundedNorm(nn.Module):
    """w * tanh(alpha * v) + b, element by element, with a scalar alpha.  Applied inside `seq_ops.bounded_sum`,
    `seq_ops.bounded_way_out` and `seq_ops.embed_bounded` (with the sum that precedes it), which take its `parts`."""

    def __init__(self, dim: int):
        super().__init__()
        self.alpha = _zeros(1, dtype=torch.float32)
        self.weight = _zeros(dim, dtype=torch.float32)
        self.bias = _zeros(dim, dtype=torch.float32)

    @property
    def parts(self):
        return self.alpha, self.weight, self.bias


class BiasedRotaryAttention(nn.Module):
    """Grouped-query softmax attention with fp32 scores over a position-addressed cache.  q, k and v have biases; the first
    `rot_dims` entries of every q and k head are turned by the position (frequencies from `rot_base` and the optional
    `rot_scaling`, whose gain multiplies the turned entries); `sink`: a learned logit per head joins the softmax denominator;
    query i sees key j <= i when `i - j < window` (window 0: every earlier key)."""

    def __init__(self, dim: int, heads: int, kv_heads: int, head_dim: int, v_dim: int, scale: float, rot_base: float, rot_dims: int,
                 rot_scaling: Optional[Dict[str, Any]], dtype, sink: bool = True, window: int = 0, interleaved: bool = True):
        super().__init__()
        if heads % kv_heads:
            raise ValueError("kv heads must divide the heads")
        if rot_dims % 2 or not 0 <= rot_dims <= head_dim:
            raise ValueError("rotary dims must be even and at most the head size")
        self.dim, self.heads, self.kv_heads, self.head_dim, self.v_dim = dim, int(heads), int(kv_heads), int(head_dim), int(v_dim)
        self.scale, self.rot_dims, self.window, self.interleaved = float(scale), int(rot_dims), int(window), bool(interleaved)
        self.nq, self.nk, self.nv = self.heads * self.head_dim, self.kv_heads * self.head_dim, self.kv_heads * self.v_dim
        self.w_in = _zeros(_pad16(self.nq + self.nk + self.nv), dim, dtype=dtype)      # rows: q | k | v | padding
        self.b_in = _zeros(self.nq + self.nk + self.nv, dtype=torch.float32)
        self.sink = _zeros(self.heads, dtype=torch.float32) if sink else None
        self.w_o = _zeros(dim, self.heads * self.v_dim, dtype=dtype)
        inv_freq, self.turn_gain = _stretched_inv_freq(rot_base, self.rot_dims, rot_scaling)
        self.register_buffer("inv_freq", inv_freq, persistent=False)

    def cache_spec(self, max_seq_length: int):
        """(strategy, slots, constructor arguments) of this mixer's cache."""
        return ("recent_global" if self.window else "full", self.window or max_seq_length,
                dict(n_heads=self.kv_heads, head_dim=self.head_dim, v_head_dim=self.v_dim))

    def core(self, hp: Tensor, ip: Tensor, cache, one_token: bool):
        """From the projection's fp32 rows to the input of the output projection [T, heads * v_dim]."""
        T, dev, dt = hp.shape[0], hp.device, self.w_o.dtype
        H, G, D, V = self.heads, self.kv_heads, self.head_dim, self.v_dim
        q = torch.empty(T, H, D, dtype=torch.float32, device=dev)
        k = torch.empty(T, G, D, dtype=dt, device=dev)
        v = torch.empty(T, G, V, dtype=dt, device=dev)
        seq_ops.qkv_rope(hp, 0, self.nq, self.nq + self.nk, H, G, D, V, None, None, 0.0, self.rot_dims, self.interleaved,
                         self.inv_freq, None, ip, q, k, v, bias=self.b_in, turn_gain=self.turn_gain)
        y = torch.empty(T, H, V, dtype=dt, device=dev)
        cache.sequence_step(q, k, v, ip, y, window=self.window, sink=self.sink,
                            sink_mode=_lib.SINK_NONE if self.sink is None else _lib.SINK_LEARNED, scale=self.scale)
        return y.view(T, H * V), None

    kernels_per_token = 4      # input product, q/k/v rows, attention + append, output product


class MatrixMemory(nn.Module):
    """Matrix memory with exponential gates.  Per head `i = cap tanh((W_i h + b_i) / cap)`, `f = logsigmoid(cap tanh((W_f h +
    b_f) / cap))`; `m' = max(f + m, i)`; `S <- exp(f + m - m') S + exp(i - m') k v^T`, n the same with k alone;
    `o = S^T q / (max(|n . q|, exp(-m')) + den_eps)` with q times dim^-1/2; o is divided by its RMS per head, times a gain of
    all heads' width, times sigmoid(W_g h), and projected.  Input rows q | k | v | g | i | f | padding.  State per sequence
    (fp32): S [heads, dim, v_dim], and per head n, m and a counter of the kernels."""

    den_eps = 1e-6

    def __init__(self, dim: int, heads: int, head_dim: int, v_dim: int, gate_cap: float, eps: float, dtype):
        super().__init__()
        if not gate_cap > 0:
            raise ValueError("the gates' soft cap must be positive")
        self.dim, self.heads, self.head_dim, self.v_dim = dim, int(heads), int(head_dim), int(v_dim)
        self.gate_cap, self.eps = float(gate_cap), float(eps)
        self.nk, self.nv = self.heads * self.head_dim, self.heads * self.v_dim
        self.w_in = _zeros(_pad16(2 * (self.nk + self.nv + self.heads)), dim, dtype=dtype)
        self.i_bias = _zeros(self.heads, dtype=torch.float32)
        self.f_bias = _zeros(self.heads, dtype=torch.float32)
        self.norm_w = _zeros(self.nv, dtype=torch.float32)
        self.w_o = _zeros(dim, self.nv, dtype=dtype)

    def cache_spec(self, max_seq_length: int):
        return "state", 0, dict(n_heads=self.heads, head_dim=self.head_dim, state_cols=self.v_dim, state_vectors=self.heads,
                                state_width=self.head_dim + 2)

    def scan(self, hp: Tensor, state) -> Tensor:
        """The recurrence over the projection's rows -> fp32 [T, heads * v_dim]."""
        o = torch.empty(hp.shape[0], self.nv, dtype=torch.float32, device=hp.device)
        H, nk, nv, g = self.heads, self.nk, self.nv, 2 * (self.nk + self.nv)
        seq_ops.mlstm(hp[:, :nk], hp[:, nk:2 * nk], hp[:, 2 * nk:2 * nk + nv], hp[:, g:g + H], hp[:, g + H:g + 2 * H], self.i_bias, self.f_bias,
                      self.gate_cap, self.head_dim ** -0.5, state.matrix, state.vectors, o, H, self.head_dim, self.v_dim, self.den_eps)
        return o

    def core(self, hp: Tensor, ip: Tensor, state, one_token: bool):
        """From the projection's fp32 rows to the input of the output projection: its rows, or for one token the recipe by
        which that product forms them itself."""
        o = self.scan(hp, state)
        gate = hp[:, 2 * self.nk + self.nv:2 * (self.nk + self.nv)]
        if one_token:
            return None, seq_ops.gated_heads_row(o, self.norm_w, gate, _lib.ACT_SIGMOID, self.eps, part=self.v_dim)
        on = torch.empty(hp.shape[0], self.nv, dtype=self.w_o.dtype, device=hp.device)
        seq_ops.gated_rms_groups(o, gate, _lib.ACT_SIGMOID, False, self.norm_w, on, self.heads, self.eps)
        return on, None

    kernels_per_token = 3      # input product, recurrence, output product with the head norm and gate


class WindowedLatentAttention(LatentAttention):
    """`detatar.LatentAttention` without a rotated part and without head gates, queries through a latent, over a window."""

    def __init__(self, dim: int, heads: int, head_dim: int, v_dim: int, q_rank: int, kv_rank: int, scale: float, window: int, eps: float, dtype):
        super().__init__(dim, int(heads), int(head_dim), 0, int(v_dim), int(q_rank), int(kv_rank), scale, 1.0, 0, eps, dtype, gated=False,
                         window=window)

    def cache_spec(self, max_seq_length: int):
        return "latent", self.window or max_seq_length, dict(n_heads=1, head_dim=self.row_width)

    def core(self, hp: Tensor, ip: Tensor, cache, one_token: bool):
        if one_token and self.absorbed_fits():
            return self.finish([hp], ip, cache), None
        return self.expanded(hp, ip, cache), None

    # input product, latent rows, query product, query through W_uk, attention over the rows (2), W_uv, output product
    kernels_per_token = 8


# --------------------------------------------------------------------------------------------- a layer

class Stream:
    """The residual stream of one step: `x` fp32 [T, E] and the copy the next product reads, which the way out of every
    sublayer renews together."""

    def __init__(self, x: Tensor, h: Tensor, mult: float, keep: bool):
        self.x, self.h, self.mult = x, h, mult
        self.first = x if keep else None      # the embedding output, when later passes add it

    def close(self, inp: Optional[Tensor], w: Tensor, out_norm: BoundedNorm, next_norm: BoundedNorm, one_token: bool, pre=None,
              built=(), add_first: bool = False, rows: Optional[Tensor] = None):
        """x += mult * out_norm(w inp) (+ the embedding output); h = next_norm(x).  One token: `inp` None takes the shared row
        `pre`, `built` = (activation, gate column, up column) forms the input of a gated unit.  `rows`: only these rows are
        wanted and x ends here."""
        x, add = self.x, (self.first if add_first else None)
        if one_token:
            h = torch.empty_like(self.h)
            x_out = torch.empty_like(x) if x is self.first else x
            post = seq_ops.bounded_way_out(x, out_norm.parts, self.mult, x_out, next_norm.parts, h, add)
            seq_ops.gemv_multi([(inp, w, None, *built)], pre=pre, post=post)
            self.x, self.h = x_out, h
            return
        y = _mm(inp, w)
        if rows is None:
            x_out, h = (torch.empty_like(x) if x is self.first else x), torch.empty_like(self.h)
        else:
            x_out, h = None, torch.empty(rows.numel(), x.shape[1], dtype=self.h.dtype, device=x.device)
        seq_ops.bounded_sum(x, y, out_norm.parts, self.mult, add, x_out, next_norm.parts, h, rows)
        self.x, self.h = x_out, h

    def add(self, next_norm: BoundedNorm):
        """x += the embedding output, on its own; h = next_norm(x)."""
        x_out = torch.empty_like(self.x) if self.x is self.first else self.x
        seq_ops.bounded_sum(self.x, add=self.first, x_out=x_out, next_norm=next_norm.parts, h=self.h)
        self.x = x_out


class RelanexBlock(nn.Module):
    """The weights of one layer: mixer and optional feed-forward, each with a norm in front and one behind."""

    def __init__(self, cfg: RelanexArgs, layer: Dict[str, Any], dtype):
        super().__init__()
        E, mlp = cfg.dim, layer.get("mlp")
        self.kind = layer["type"]
        self.mixer = self.make_mixer(cfg, layer, dtype, int(layer["mixer"].get("q_rank", 1)))
        self.norm1, self.norm1b = BoundedNorm(E), BoundedNorm(E)
        self.mlp = self.w_gu = self.norm2 = self.norm2b = None
        if mlp:
            self.mlp = GatedMLP(E, int(mlp["ff"]), _lib.ACT_SILU, dtype)
            self.w_gu = _zeros(2 * self.mlp.ff, E, dtype=dtype)      # rows: gate | up
            self.norm2, self.norm2b = BoundedNorm(E), BoundedNorm(E)

    @staticmethod
    def make_mixer(cfg: RelanexArgs, layer: Dict[str, Any], dtype, q_rank: int):
        E, m = cfg.dim, layer["mixer"]
        heads, dim = int(m["heads"]), int(m["dim"])
        vdim, window = int(m.get("vdim", dim)), int((m.get("mask") or {}).get("size", 0))
        scale = float(m.get("scale", dim ** -0.5))
        if layer["type"] == "attention":
            rot = m.get("rot") or {}
            return BiasedRotaryAttention(E, heads, int(m.get("kv_heads", heads)), dim, vdim, scale, float(rot.get("base", 10000.0)),
                                         int(rot.get("dims", 0)), rot.get("scaling"), dtype, window=window)
        if layer["type"] == "latent_attention":
            return WindowedLatentAttention(E, heads, dim, vdim, q_rank, int(m["kv_rank"]), scale, window, cfg.norm_eps, dtype)
        return MatrixMemory(E, heads, dim, vdim, float(m["gate_cap"]), cfg.norm_eps, dtype)

    def forward(self, s: Stream, ip: Tensor, store, next_norm: BoundedNorm, one_token: bool, add_first: bool = False,
                rows: Optional[Tensor] = None):
        """Runs the layer on s.h = norm1(s.x); `next_norm` reads what comes after it (with the embedding output added when
        the next pass starts there)."""
        m, last = self.mixer, dict(add_first=add_first, rows=rows)
        inp, pre = m.core(_product(s.h, m.w_in, one_token), ip, store, one_token)
        s.close(inp, m.w_o, self.norm1b, next_norm if self.mlp is None else self.norm2, one_token, pre=pre, **(last if self.mlp is None else {}))
        if self.mlp is None:
            return
        f = self.mlp
        gu = _product(s.h, self.w_gu, one_token)
        if one_token:
            s.close(gu, f.w_down, self.norm2b, next_norm, True, built=(f.act, 0, f.ff), **last)
            return
        act = torch.empty(gu.shape[0], f.ff, dtype=f.w_down.dtype, device=gu.device)
        seq_ops.gated_unit(gu, 0, f.ff, act, f.act)
        s.close(act, f.w_down, self.norm2b, next_norm, False, **last)

    def kernels_per_token(self) -> int:
        return self.mixer.kernels_per_token + (2 if self.mlp is not None else 0)


class RelanexLayer(nn.Module):
    """One run of a block: the (possibly shared) weights with this run's own cache or state; `starts_pass`: the embedding
    output is added to the stream before it."""

    def __init__(self, block: RelanexBlock, shares_weights: bool, starts_pass: bool):
        super().__init__()
        if shares_weights:
            object.__setattr__(self, "block", block)    # not registered twice
        else:
            self.block = block
        self.starts_pass = starts_pass
        self.store = None


# --------------------------------------------------------------------------------------------- the model

class RelanexTransformer(nn.Module):
    """Same runtime surface as `model.Transformer`: setup_caches / reset_caches / forward / min_cache_length /
    get_cache_stats / prompt_cache_overflow, `config.block_size`, `config.n_layer` (the number of layer runs)."""

    supports_prompt_portions = True

    def __init__(self, config: RelanexArgs, dtype=torch.bfloat16):
        super().__init__()
        assert dtype in (torch.bfloat16, torch.float32)
        self.config, self.dtype = config, dtype
        self.tok_embeddings = _zeros(config.vocab_size, config.dim, dtype=dtype)
        self.embed_norm = BoundedNorm(config.dim)
        blocks: Dict[int, RelanexBlock] = {}
        layers = []
        for i, t in config.runs():
            fresh = i not in blocks
            if fresh:
                blocks[i] = RelanexBlock(config, config.layers[i], dtype)
            layers.append(RelanexLayer(blocks[i], not fresh, bool(t) and i == config.loop_start))
        self.layers = nn.ModuleList(layers)
        self.norm = BoundedNorm(config.dim)
        self.output = _zeros(config.vocab_size, config.dim, dtype=dtype)
        self.max_batch_size = 1
        self.max_seq_length = 0
        # one-token steps through this package's product kernels and the absorbed latent attention; False = the kernels of a
        # prompt portion of one token (library products), used by A/B tests
        self.fused_decode = True

    def blocks(self):
        """(layer index in the configuration, block) of every distinct block, in running order."""
        seen, out = set(), []
        for (i, _), layer in zip(self.config.runs(), self.layers):
            if i not in seen:
                seen.add(i)
                out.append((i, layer.block))
        return out

    # ---- caches and state -------------------------------------------------------------------------
    def layer_cache_plan(self, cache_kwargs: Dict[str, Any], max_seq_length: int) -> Dict[str, Any]:
        """Per layer run: "full" rows for attention, "latent" rows for latent attention (a ring of one window), "state" for a
        matrix memory."""
        ck = dict(cache_kwargs or {})
        ck["max_seq_length"] = max_seq_length
        specs = [l.block.mixer.cache_spec(max_seq_length) for l in self.layers]
        ck["cache_strategy"], ck["max_cache_length"] = [s[0] for s in specs], [s[1] for s in specs]
        ck["global_tokens"] = 0
        ck["cache_bits"] = None
        ck["prompt_compression_strategy"] = ["none"] * len(self.layers)
        return ck

    def setup_caches(self, **kwargs):
        lengths, max_seq_length = kwargs["max_cache_length"], kwargs.get("max_seq_length")
        for i, layer in enumerate(self.layers):
            strategy = kwargs["cache_strategy"][i]
            ctor, _ = get_cache_constructor(strategy)
            spec = dict(layer.block.mixer.cache_spec(int(max_seq_length or 0))[2])
            if strategy != "state":
                spec.update(dtype=self.dtype, max_cache_length=int(lengths[i]), max_seq_length=max_seq_length, global_tokens=0, cache_bits=None)
            layer.store = ctor(self.max_batch_size, **spec)
        self.max_seq_length = int(max_seq_length or max(lengths))

    def reset_caches(self):
        """Gives back what the finished sequence held: every slot empty, every state zero."""
        for layer in self.layers:
            layer.store.reset()

    def _unwindowed(self):
        return [l.block.kind != "mlstm" and not l.block.mixer.window for l in self.layers]

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
        state that earlier steps left.  `collect`, if a list, receives the residual stream after every layer run."""
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
        rows = None
        if not one:
            rows = torch.full((1,), T - 1, dtype=torch.int64, device=dev) if logits_at is None else \
                logits_at.to(device=dev, dtype=torch.int64).contiguous()
        x, h = torch.empty(T, E, dtype=torch.float32, device=dev), torch.empty(T, E, dtype=dt, device=dev)
        seq_ops.embed_bounded(tokens, self.tok_embeddings, self.embed_norm.parts, x, self.layers[0].block.norm1.parts, h)
        s = Stream(x, h, self.config.residual_mult, any(l.starts_pass for l in self.layers))
        for layer, nxt in zip(self.layers, [*self.layers[1:], None]):
            next_norm = self.norm if nxt is None else nxt.block.norm1
            again = nxt is not None and nxt.starts_pass
            layer.block(s, ip, layer.store, next_norm, one, add_first=again and collect is None,
                        rows=rows if nxt is None and collect is None else None)
            if collect is not None:
                collect.append(s.x.clone())
                if again:
                    s.add(next_norm)
        if collect is not None and rows is not None:
            s.h = s.h[rows]
        return _product(s.h, self.output, one).view(1, s.h.shape[0], -1)

    def kernels_per_token(self) -> int:
        """Launches of this package's kernels in one decode step (fused_decode)."""
        return 2 + sum(l.block.kernels_per_token() for l in self.layers)   # embedding row, head

    # ---- weights --------------------------------------------------------------------------------
    def load_tensors(self, tensors: Dict[str, Tensor]):
        """Fills the parameters from the checkpoint's tensor names ('embed', 'embed.norm', 'l<i>.norm1' / '.norm1b' / '.norm2' /
        '.norm2b', each norm with '.alpha' and '.b', 'l<i>.mix.*', 'l<i>.mlp.*', 'final.norm', 'head'), fusing the projection
        rows that read the same input."""
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

        def put_norm(norm, name):
            put(norm.weight, get(name, (E,)))
            put(norm.bias, get(name + ".b", (E,)))
            alpha = get(name + ".alpha")
            if alpha.numel() != 1:
                raise ValueError(f"{name}.alpha: shape {tuple(alpha.shape)} is not a scalar")
            put(norm.alpha, alpha)

        put(self.tok_embeddings, get("embed", (cfg.vocab_size, E)))
        put_norm(self.embed_norm, "embed.norm")
        for i, b in self.blocks():
            p, q = f"l{i}.", f"l{i}.mix."
            put_norm(b.norm1, p + "norm1")
            put_norm(b.norm1b, p + "norm1b")
            m = b.mixer
            if b.kind == "attention":
                put(m.w_in, _padded_rows([get(q + "q", (m.nq, E)), get(q + "k", (m.nk, E)), get(q + "v", (m.nv, E))], m.w_in.shape[0]))
                put(m.b_in, torch.cat([get(q + "q.b", (m.nq,)), get(q + "k.b", (m.nk,)), get(q + "v.b", (m.nv,))]))
                put(m.sink, get(q + "sink", (m.heads,)))
                put(m.w_o, get(q + "o", (E, m.heads * m.v_dim)))
            elif b.kind == "latent_attention":
                layer = cfg.layers[i]
                if "q_rank" not in layer["mixer"]:      # then the query latent's size is a tensor shape
                    m = b.mixer = RelanexBlock.make_mixer(cfg, layer, self.dtype, get(q + "dq").shape[0]).to(m.w_in.device)
                H, D, V, C, R = m.heads, m.head_dim, m.v_dim, m.kv_rank, m.q_rank
                put(m.w_in, _padded_rows([get(q + "dq", (R, E)), get(q + "dkv", (C, E))], m.w_in.shape[0]))
                put(m.q_norm, get(q + "dq.norm", (R,)))
                put(m.kv_norm, get(q + "dkv.norm", (C,)))
                put(m.w_uq, get(q + "uq", (H * D, R)))
                uk, uv = get(q + "uk", (H * D, C)), get(q + "uv", (H * V, C))
                put(m.w_ukv, torch.cat([uk, uv]))
                put(m.w_uk_t, uk.reshape(H, D, C).transpose(1, 2))
                put(m.w_o, get(q + "o", (E, H * V)))
            else:
                H, nk, nv = m.heads, m.nk, m.nv
                put(m.w_in, _padded_rows([get(q + n, (w, E)) for n, w in (("q", nk), ("k", nk), ("v", nv), ("g", nv), ("i", H), ("f", H))],
                                         m.w_in.shape[0]))
                put(m.i_bias, get(q + "i.b", (H,)))
                put(m.f_bias, get(q + "f.b", (H,)))
                put(m.norm_w, get(q + "norm", (nv,)))
                put(m.w_o, get(q + "o", (E, nv)))
            f = b.mlp
            if f is not None:
                q = p + "mlp."
                put_norm(b.norm2, p + "norm2")
                put_norm(b.norm2b, p + "norm2b")
                put(b.w_gu, torch.cat([get(q + "gate", (f.ff, E)), get(q + "up", (f.ff, E))]))
                put(f.w_down, get(q + "down", (E, f.ff)))
        put_norm(self.norm, "final.norm")
        put(self.output, get("head", (cfg.vocab_size, E)))
        return sorted(set(tensors) - used)

    @classmethod
    def from_config(cls, cfg: Dict[str, Any], dtype=torch.bfloat16):
        return cls(RelanexArgs.from_config(cfg), dtype)
