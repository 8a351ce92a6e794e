"""Legavik: a pre-norm decoder whose norms compute no statistics (a learned tanh), with grouped-query window attention that keeps the
sequence's first tokens in sight, layers that run full-length attention and a gated delta rule side by side, and routed experts.

With x the float32 residual stream and T(v; n) = tanh(n.alpha * v) * n + n.b:

    x = embed[token]
    x <- x + mixer(T(x; norm1));      x <- x + ff(T(x; norm2))                     (a layer may have no feed-forward)
    logits = cap * tanh(head T(x; final.norm) / cap)

mixers (`layers[i].type`):
    attention   q = W_q h, k = W_k h, the values are k as projected. q and k are rotated (the first `rot.dims` entries of a head, entry i
                with i + dims/2, frequencies stretched and the pair scaled by an amplitude as `rot.scaling` says), then made unit-RMS
                per head. Position i sees j when i - j < mask.size or j < mask.keep_first. Head output * sigmoid(W_g h)_head, W_o.
    parallel    left_scale * left + right_scale * right of the same h:
      left      q, k, v with biases, each through a short causal convolution; q, k unit-RMS per head times a shared weight; q times
                1 + coef * ln(floor((p + 1) / every) + 1); causal over the whole sequence; one gate per head; W_o with a bias.
      right     q, k (kv_heads x dim), v (heads x vdim) through a convolution and silu; q, k unit vectors (q times dim^-1/2); decays per
                head and key channel g = exp(-exp(A_log) softplus(W_a2 W_a1 h + dt_bias)); S <- g S, u = beta (v - S^T k),
                S <- S + k u^T, o = S^T q with beta = sigmoid(W_b h); o unit-RMS per head * norm * sigmoid(W_g2 W_g1 h); W_o.
feed-forward (`mlp.kind` = moe): s = softmax(W_router h) in float32; the experts form groups of neighbours, a group scores its largest s,
    only the best groups stay; the `top` largest s, divided by their sum, weight expert(h) = W_down (silu(W_gate h) * W_up h).

Wiring follows `kinanex.KinanexModel`: a flat token batch with per-token slot and position (`state.BatchMeta`), state held by the model
and indexed by slot, a scratch arena allocated once, dense products in the vendor library, everything else in the sequence-mixer
kernel library (`ops.seq_*`, `ops.moe_*`). One product makes everything a mixer reads from h, one product closes it (the two halves of
a parallel layer write side by side, already scaled). Every residual sum is fused with the norm that follows it
(`ops.seq_residual_tanh`). Per-slot state: key / value rows of every attention (window layers in rings whose first rows are pinned), the
float32 matrices of the delta rule, and the last `conv - 1` inputs of every convolution (double-buffered by the step's phase). Nothing is
cleared when a slot is released: cache rows are valid by position, and the recurrence starts from zero at position 0.
"""
from __future__ import annotations

import copy
import json
import math
import os
from dataclasses import dataclass, field
from typing import Dict, List, Optional

import torch

from . import ops
from .seq_layers import PROMPT_TILES_MIN_CTAS, TILES_MIN_TOKENS, attend_window, run_experts
from .state import SCAN_SHORT, BatchMeta

UNIT_EPS = 1e-6                     # under the root of the delta rule's unit vectors
GROUP_TOP = 1                       # a group's score is its largest expert score
FULL_WINDOW = 1 << 30               # attention over the whole sequence: a window no sequence reaches


@dataclass
class LegavikAttention:
    """The attention mixer, or the left half of a parallel one."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int] = None    # None: the whole sequence
    keep_first: int = 0
    rot_dims: int = 0
    rot_base: float = 10000.0
    rot_scaling: Optional[Dict[str, float]] = None      # factor, original, fast, slow
    conv: int = 1                   # left half: taps of the convolution ...
    temp_coef: float = 0.0
    temp_every: int = 0             # 0: no temperature


@dataclass
class LegavikDelta:
    """The right half of a parallel mixer."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    decay_rank: int = 0             # inner sizes of the decay and gate projections: the checkpoint's tensors give them
    gate_rank: int = 0


@dataclass
class LegavikMixer:
    kind: str                       # "attention" | "parallel"
    att: LegavikAttention
    delta: Optional[LegavikDelta] = None
    left_scale: float = 1.0
    right_scale: float = 1.0


@dataclass
class LegavikFF:
    ff: int                         # hidden size of one expert
    experts: int
    top: int
    groups: int = 1
    keep: int = 1


@dataclass
class LegavikLayer:
    mixer: LegavikMixer
    mlp: Optional[LegavikFF]


def rotary_frequencies(dims: int, base: float, scaling: Optional[Dict[str, float]] = None) -> torch.Tensor:
    """f_i = base^(-2i / dims), i < dims / 2 (float64). With `scaling` = {factor, original, fast, slow}: the pair that turns r times within
    `original` positions has the index dims * ln(original / (2 pi r)) / (2 ln base); pairs up to the index of `fast` turns (rounded
    down, at least 0) keep f, pairs from the index of `slow` turns on (rounded up, at most dims - 1) get f / factor, a ramp between."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    f = torch.tensor(float(base), dtype=torch.float64) ** (-2.0 * i / max(dims, 1))
    if scaling and dims:
        factor, orig, fast, slow = (float(scaling[k]) for k in ("factor", "original", "fast", "slow"))
        index = lambda turns: dims * math.log(orig / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
        lo, hi = max(math.floor(index(fast)), 0), min(math.ceil(index(slow)), dims - 1)
        ramp = torch.clamp((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
        f = f / factor * ramp + f * (1.0 - ramp)
    return f


def rotary_amplitude(scaling: Optional[Dict[str, float]]) -> float:
    return 0.1 * math.log(float(scaling["factor"])) + 1.0 if scaling else 1.0


def _attention_from(m: dict, i: int) -> LegavikAttention:
    rot, mask, temp = m.get("rot") or {}, m.get("mask") or {}, m.get("q_temp") or {}
    heads, dim = int(m["heads"]), int(m["dim"])
    a = LegavikAttention(heads=heads, kv_heads=int(m.get("kv_heads", heads)), dim=dim, vdim=int(m.get("vdim", dim)), scale=float(m["scale"]),
                         window=int(mask["size"]) if mask.get("size") else None, keep_first=int(mask.get("keep_first", 0)),
                         rot_dims=int(rot.get("dims", 0)), rot_base=float(rot.get("base", 10000.0)),
                         rot_scaling=dict(rot["scaling"]) if rot.get("scaling") else None, conv=int(m.get("conv", 1)),
                         temp_coef=float(temp.get("coef", 0.0)), temp_every=int(temp.get("every", 0)))
    if a.kv_heads < 1 or a.heads % a.kv_heads:
        raise ValueError(f"layer {i}: {a.heads} heads over {a.kv_heads} key heads")
    if a.rot_dims % 2 or a.rot_dims > a.dim:
        raise ValueError(f"layer {i}: {a.rot_dims} rotated dimensions of {a.dim}")
    if a.conv < 1 or (a.window is not None and a.window < 1) or a.keep_first < 0:
        raise ValueError(f"layer {i}: a convolution of {a.conv} taps, a window of {a.window}, {a.keep_first} kept tokens")
    return a


@dataclass
class LegavikConfig:
    vocab: int
    width: int
    eps: float
    logit_softcap: Optional[float] = None
    layers: List[LegavikLayer] = field(default_factory=list)
    name: str = "legavik"

    @staticmethod
    def from_dict(d: dict) -> "LegavikConfig":
        layers = []
        for i, e in enumerate(d["layers"]):
            kind, m = e.get("type"), e["mixer"]
            if kind == "attention":
                mixer = LegavikMixer(kind=kind, att=_attention_from(m, i))
                if mixer.att.vdim != mixer.att.dim:
                    raise ValueError(f"layer {i}: the values are the keys, but their sizes are {mixer.att.vdim} and {mixer.att.dim}")
            elif kind == "parallel":
                r = m["right"]
                dl = LegavikDelta(heads=int(r["heads"]), kv_heads=int(r.get("kv_heads", r["heads"])), dim=int(r["dim"]),
                                  vdim=int(r.get("vdim", r["dim"])), conv=int(r["conv"]))
                if dl.kv_heads < 1 or dl.heads % dl.kv_heads or dl.conv < 1:
                    raise ValueError(f"layer {i}: {dl.heads} heads over {dl.kv_heads} key heads, a convolution of {dl.conv} taps")
                mixer = LegavikMixer(kind=kind, att=_attention_from(m["left"], i), delta=dl, left_scale=float(m.get("left_scale", 1.0)),
                                     right_scale=float(m.get("right_scale", 1.0)))
            else:
                raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
            f = e.get("mlp")
            if f is None:
                mlp = None
            elif f.get("kind", "moe") == "moe":
                r = f["router"]
                g = r.get("groups") or {}
                count = int(g.get("count", 1))
                mlp = LegavikFF(ff=int(f["expert"]["ff"]), experts=int(r["experts"]), top=int(r["top"]), groups=count,
                                keep=int(g.get("keep", count)))
                if mlp.groups < 1 or mlp.experts % mlp.groups or not 1 <= mlp.keep <= mlp.groups:
                    raise ValueError(f"layer {i}: {mlp.experts} experts in {mlp.groups} groups, keep {mlp.keep}")
                if not 1 <= mlp.top <= mlp.keep * (mlp.experts // mlp.groups):
                    raise ValueError(f"layer {i}: top {mlp.top} of {mlp.keep} groups of {mlp.experts // mlp.groups} experts")
            else:
                raise ValueError(f"layer {i}: unknown feed-forward kind {f.get('kind')!r}")
            layers.append(LegavikLayer(mixer=mixer, mlp=mlp))
        cap = d.get("logit_softcap")
        return LegavikConfig(vocab=int(d["vocab"]), width=int(d["width"]), eps=float(d["norm"]["eps"]),
                             logit_softcap=float(cap) if cap else None, layers=layers)

    def to_dict(self) -> dict:
        out = {"architecture": "Legavik", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps}, "layers": []}
        if self.logit_softcap:
            out["logit_softcap"] = self.logit_softcap

        def att(a):
            mx = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale}
            if a.window is not None:
                mx["mask"] = {"size": a.window, "keep_first": a.keep_first}
            if a.rot_dims:
                mx["rot"] = {"base": a.rot_base, "dims": a.rot_dims}
                if a.rot_scaling:
                    mx["rot"]["scaling"] = dict(a.rot_scaling)
            if a.temp_every:
                mx["q_temp"] = {"coef": a.temp_coef, "every": a.temp_every}
            return mx

        for l in self.layers:
            m, f = l.mixer, l.mlp
            mx = att(m.att)
            if m.kind == "parallel":
                mx["conv"] = m.att.conv
                dl = m.delta
                mx = {"left": mx, "right": {"heads": dl.heads, "kv_heads": dl.kv_heads, "dim": dl.dim, "vdim": dl.vdim, "conv": dl.conv},
                      "left_scale": m.left_scale, "right_scale": m.right_scale}
            out["layers"].append({"type": m.kind, "mixer": mx, "mlp": None if f is None else
                                  {"kind": "moe", "expert": {"ff": f.ff},
                                   "router": {"experts": f.experts, "top": f.top, "groups": {"count": f.groups, "keep": f.keep}}}})
        return out

    def with_ranks(self, weights: Optional[Dict[str, torch.Tensor]] = None, decay_rank: int = 0, gate_rank: int = 0) -> "LegavikConfig":
        """A copy whose delta halves have their inner projection sizes filled in: from a checkpoint's tensors, or as given (for random
        weights; at least 1)."""
        cfg = copy.deepcopy(self)
        for i, l in enumerate(cfg.layers):
            if l.mixer.delta is None:
                continue
            for attr, name, given in (("decay_rank", "a1", decay_rank), ("gate_rank", "g1", gate_rank)):
                key = f"l{i}.mix.right.{name}"
                if weights is not None:
                    if key not in weights:
                        raise KeyError(f"tensor {key} is missing from the checkpoint")
                    given = int(weights[key].shape[0])
                setattr(l.mixer.delta, attr, max(given, 1))
        return cfg

    def tensor_shapes(self) -> Dict[str, tuple]:
        """Name -> shape of every tensor a checkpoint of this configuration must hold (the inner sizes of the decay and gate
        projections filled in by `with_ranks`)."""
        W = self.width
        out = {"embed": (self.vocab, W)}

        def norm(name):
            out.update({name: (W,), name + ".b": (W,), name + ".alpha": ()})

        for i, l in enumerate(self.layers):
            m, f, p = l.mixer, l.mlp, f"l{i}."
            a, dl = m.att, m.delta
            norm(p + "norm1")
            x = p + "mix."
            if m.kind == "attention":
                out.update({x + "q": (a.heads * a.dim, W), x + "k": (a.kv_heads * a.dim, W), x + "g": (a.heads, W), x + "o": (W, a.heads * a.vdim)})
            else:
                y = x + "left."
                for n, rows in (("q", a.heads * a.dim), ("k", a.kv_heads * a.dim), ("v", a.kv_heads * a.vdim)):
                    out.update({y + n: (rows, W), y + n + ".b": (rows,), y + n + ".conv": (rows, a.conv)})
                out.update({y + "q.norm": (a.dim,), y + "k.norm": (a.dim,), y + "g": (a.heads, W), y + "o": (W, a.heads * a.vdim), y + "o.b": (W,)})
                y = x + "right."
                for n, rows in (("q", dl.kv_heads * dl.dim), ("k", dl.kv_heads * dl.dim), ("v", dl.heads * dl.vdim)):
                    out.update({y + n: (rows, W), y + n + ".conv": (rows, dl.conv)})
                out.update({y + "b": (dl.heads, W), y + "A_log": (dl.heads,), y + "norm": (dl.vdim,), y + "a1": (dl.decay_rank, W),
                            y + "a2": (dl.heads * dl.dim, dl.decay_rank), y + "dt_bias": (dl.heads * dl.dim,), y + "g1": (dl.gate_rank, W),
                            y + "g2": (dl.heads * dl.vdim, dl.gate_rank), y + "o": (W, dl.heads * dl.vdim)})
            if f is not None:
                norm(p + "norm2")
                y = p + "mlp."
                out[y + "router"] = (f.experts, W)
                for e in range(f.experts):
                    out.update({y + f"e{e}.gate": (f.ff, W), y + f"e{e}.up": (f.ff, W), y + f"e{e}.down": (W, f.ff)})
        norm("final.norm")
        out["head"] = (self.vocab, W)
        return out


def random_weights(cfg: LegavikConfig, seed: int = 0) -> Dict[str, torch.Tensor]:
    """Random bfloat16 tensors of a configuration (CPU): matrices ~ N(0, 1/fan_in), norm weights near 1, tanh slopes around 0.6, decays
    and step sizes in the range where the state neither dies nor saturates."""
    if any(l.mixer.delta is not None and not l.mixer.delta.decay_rank for l in cfg.layers):
        raise ValueError("random_weights: the inner projection sizes are open (LegavikConfig.with_ranks)")
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in cfg.tensor_shapes().items():
        if name.endswith(".alpha"):
            t = 0.4 + 0.4 * torch.rand(shape, generator=g)
        elif name.endswith("A_log"):
            t = 0.5 * torch.randn(shape, generator=g)
        elif len(shape) == 2:
            t = torch.randn(shape, generator=g) / shape[1] ** 0.5
        elif name.endswith(("norm1", "norm2", ".norm")):
            t = 1.0 + 0.1 * torch.randn(shape, generator=g)
        elif name.endswith("dt_bias"):
            t = -1.0 + 0.5 * torch.randn(shape, generator=g)
        else:
            t = 0.1 * torch.randn(shape, generator=g)
        out[name] = t.to(torch.bfloat16)
    return out


class _TanhNorm:
    def __init__(self, sd, name, device):
        f = dict(device=device, dtype=torch.float32)
        self.alpha = float(sd[name + ".alpha"].to(torch.float32))
        self.w, self.b = sd[name].to(**f).contiguous(), sd[name + ".b"].to(**f).contiguous()


class _LayerWeights:
    """Device tensors of one layer: large matrices in the activation type (everything that reads the mixer's input in one, the output
    matrices of a parallel layer side by side), vectors, convolutions, the router and everything the recurrence reads in float32."""

    def __init__(self, cfg: LegavikConfig, i: int, sd: Dict[str, torch.Tensor], dtype, device):
        spec, p = cfg.layers[i], f"l{i}."
        m, f = spec.mixer, spec.mlp
        a, dl = m.att, m.delta

        def big(*names, dim=0):
            t = torch.cat([sd[p + n] for n in names], dim) if len(names) > 1 else sd[p + names[0]]
            return t.to(device=device, dtype=dtype).contiguous()

        def small(*names):
            t = torch.cat([sd[p + n].to(torch.float32) for n in names], 0) if len(names) > 1 else sd[p + names[0]]
            return t.to(device=device, dtype=torch.float32).contiguous()

        self.norm1 = _TanhNorm(sd, p + "norm1", device)
        self.inv_freq = rotary_frequencies(a.rot_dims, a.rot_base, a.rot_scaling).to(device=device, dtype=torch.float32) if a.rot_dims else None
        self.rot_amp = rotary_amplitude(a.rot_scaling)
        if m.kind == "attention":
            self.w_in = big("mix.q", "mix.k", "mix.g")                                            # rows [q ; k ; one gate per head]
            self.o = big("mix.o")
        else:
            L, R = "mix.left.", "mix.right."
            parts = [L + "q", L + "k", L + "v", R + "q", R + "k", R + "v", R + "a1", R + "g1", L + "g", R + "b"]
            self.w_in = big(*parts)
            bias = torch.zeros(self.w_in.shape[0], dtype=torch.float32)
            left = torch.cat([sd[p + L + n + ".b"].to(torch.float32) for n in "qkv"])
            bias[:left.numel()] = left
            self.b_in = bias.to(device=device, dtype=dtype)
            self.conv_l = small(L + "q.conv", L + "k.conv", L + "v.conv").t().contiguous()       # [taps, channels]
            self.conv_r = small(R + "q.conv", R + "k.conv", R + "v.conv").t().contiguous()
            self.q_norm, self.k_norm = small(L + "q.norm"), small(L + "k.norm")
            self.o = big(L + "o", R + "o", dim=1)                                                 # columns [left heads | right heads]
            self.o_b = (small(L + "o.b") * m.left_scale).contiguous()
            self.a2, self.g2 = big(R + "a2"), big(R + "g2")
            self.A_log, self.dt_bias, self.r_norm = small(R + "A_log"), small(R + "dt_bias"), small(R + "norm")
        if f is not None:
            self.norm2 = _TanhNorm(sd, p + "norm2", device)
            self.router = small("mlp.router")
            self.gate_up = torch.stack([torch.cat([sd[p + f"mlp.e{e}.gate"], sd[p + f"mlp.e{e}.up"]], 0) for e in range(f.experts)]) \
                .to(device=device, dtype=dtype).contiguous()                                      # [E, 2 F, W], gate rows first
            self.edown = torch.stack([sd[p + f"mlp.e{e}.down"] for e in range(f.experts)]).to(device=device, dtype=dtype).contiguous()


class LegavikModel(torch.nn.Module):
    """Weights, per-slot state and the forward pass over a flat token batch (`state.BatchMeta`).

    dtype: torch.bfloat16 (serving: bfloat16 matrix products with float32 accumulation) or torch.float32 (everything in true
    float32). n_slots sequences can be live at once; a step carries at most max_step_tokens tokens; a sequence holds at most
    max_seq_tokens tokens where a layer attends over all of it (such caches have that many rows per slot; window layers keep their
    first rows and a ring of window - 1 + max_step_tokens)."""

    architecture = "Legavik"
    DEFAULT_SEQ_TOKENS = 8192

    def __init__(self, cfg: LegavikConfig, weights: Dict[str, torch.Tensor], dtype=torch.bfloat16, device="cuda",
                 n_slots: int = 8, max_step_tokens: int = 2048, max_seq_tokens: Optional[int] = None):
        super().__init__()
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("LegavikModel: dtype must be torch.bfloat16 or torch.float32")
        cfg = cfg.with_ranks(weights)
        for name, shape in cfg.tensor_shapes().items():
            if name not in weights:
                raise KeyError(f"tensor {name} is missing from the checkpoint")
            if tuple(weights[name].shape) != tuple(shape):
                raise ValueError(f"tensor {name}: shape {tuple(weights[name].shape)}, the configuration says {tuple(shape)}")
        self.cfg, self.dtype, self.device = cfg, dtype, torch.device(device)
        self.n_slots, self.max_step_tokens = n_slots, max_step_tokens
        # true float32 products in float32 mode; no reduced-precision accumulation of bfloat16 products
        torch.backends.cuda.matmul.allow_tf32 = False
        torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
        dev, W, T = self.device, cfg.width, max_step_tokens
        f32 = dict(dtype=torch.float32, device=dev)
        act = dict(dtype=dtype, device=dev)
        self.embed = weights["embed"].to(**act).contiguous()
        self.head = weights["head"].to(**act).contiguous()
        self.final_norm = _TanhNorm(weights, "final.norm", dev)
        self.weights = [_LayerWeights(cfg, i, weights, dtype, dev) for i in range(len(cfg.layers))]
        # ---- per-slot state ----
        limit = max(int(max_seq_tokens or self.DEFAULT_SEQ_TOKENS), 1)
        rows: Dict[int, int] = {}
        bounded = False                                                                        # whether a cache bounds the sequence length
        for i, l in enumerate(cfg.layers):
            a = l.mixer.att
            ring = limit if a.window is None else a.keep_first + a.window - 1 + T
            rows[i] = max(min(ring, limit), a.keep_first + 1)
            bounded |= rows[i] < ring or a.window is None
        self.max_seq_len = limit if bounded else None                                          # checked by the scheduler
        self.cache_k: Dict[int, torch.Tensor] = {}                                             # layer -> [slots, rows, G, D]
        self.cache_v: Dict[int, torch.Tensor] = {}                                             # layer -> [slots, rows, G, DV]
        self.rec_state: Dict[int, torch.Tensor] = {}                                           # layer -> float32 [slots, H, D, DV]
        self.tail_l: Dict[int, torch.Tensor] = {}                                              # layer -> float32 [2, slots, taps - 1, C]
        self.tail_r: Dict[int, torch.Tensor] = {}
        mix = [l.mixer for l in cfg.layers]
        for i, m in enumerate(mix):
            a, dl = m.att, m.delta
            self.cache_k[i] = torch.zeros(n_slots, rows[i], a.kv_heads, a.dim, **act)
            self.cache_v[i] = torch.zeros(n_slots, rows[i], a.kv_heads, a.vdim, **act)
            if dl is not None:
                self.tail_l[i] = torch.zeros(2, n_slots, a.conv - 1, (a.heads + a.kv_heads) * a.dim + a.kv_heads * a.vdim, **f32)
                self.tail_r[i] = torch.zeros(2, n_slots, dl.conv - 1, 2 * dl.kv_heads * dl.dim + dl.heads * dl.vdim, **f32)
                self.rec_state[i] = torch.zeros(n_slots, dl.heads, dl.dim, dl.vdim, **f32)
        # ---- scratch arena, allocated once ----
        mx = lambda vals: max(list(vals) + [1])
        par = [m.delta for m in mix if m.delta is not None]
        ffs = [l.mlp for l in cfg.layers if l.mlp]
        self.buf_x = torch.empty(T * W, **f32)                                                 # residual stream (updated in place)
        self.buf_h = torch.empty(T * W, **act)                                                 # sublayer input
        self.buf_y = torch.empty(T * W, **act)                                                 # sublayer output
        self.buf_proj = torch.empty(T * mx(w.w_in.shape[0] for w in self.weights), **act)
        self.buf_q = torch.empty(T * mx(m.att.heads * m.att.dim for m in mix), **f32)          # normed, rotated queries
        self.buf_att = torch.empty(T * mx(w.o.shape[1] for w in self.weights), **act)          # gated head outputs
        self.buf_decay = torch.empty(T * mx(d.heads * d.dim for d in par), **f32)
        self.buf_gate = torch.empty(T * mx(d.heads * d.vdim for d in par), **act)
        blocks = max(T // SCAN_SHORT, 1)                                                       # ceil(n / 16) <= n / 8 for every segment that has blocks
        self.scan_scratch = torch.empty(mx([ops.seq_delta_channel_scratch_bytes(blocks, T, d.heads, d.dim, d.vdim) for d in par]),
                                        dtype=torch.uint8, device=dev)
        tops = mx(f.top for f in ffs)
        self.buf_idx = torch.empty(T * tops, dtype=torch.int32, device=dev)
        self.buf_rw = torch.empty(T * tops, **f32)
        self.buf_pair = torch.empty(T * tops * W if ffs else 1, **act)
        # bfloat16 takes the tensor-core forms where the sizes allow (as in repepel.RepepelModel); QSPEC_SEQ_TILES=0 keeps the plain ones
        self.use_tiles = dtype == torch.bfloat16 and os.environ.get("QSPEC_SEQ_TILES", "1") != "0"
        self.tiles_min_tokens, self.prompt_tiles_min_ctas = TILES_MIN_TOKENS, PROMPT_TILES_MIN_CTAS
        self._mm_f32_out = None              # whether torch.mm takes bfloat16 operands with a float32 out (probed once)

    # ------------------------------------------------------------------------------------------
    @classmethod
    def from_pretrained(cls, path: str, dtype=torch.bfloat16, device="cuda", **kw) -> "LegavikModel":
        from .checkpoint import read_safetensors_file
        with open(os.path.join(path, "config.json")) as f:
            cfg = LegavikConfig.from_dict(json.load(f))
        return cls(cfg, read_safetensors_file(os.path.join(path, "model.safetensors")), dtype=dtype, device=device, **kw)

    @property
    def vocab_size(self) -> int:
        return self.cfg.vocab

    def state_bytes_per_slot(self) -> int:
        ts = [t for d in (self.cache_k, self.cache_v, self.rec_state, self.tail_l, self.tail_r) for t in d.values()]
        return sum(t.numel() * t.element_size() // self.n_slots for t in ts)

    def _mm_to_f32(self, a: torch.Tensor, b_t: torch.Tensor, out: torch.Tensor) -> None:
        """out (float32) = a @ b_t^T, accumulated in float32 whatever the operands' type."""
        if a.dtype == torch.float32:
            torch.matmul(a, b_t.t(), out=out)
            return
        if self._mm_f32_out is None:
            try:
                torch.mm(a, b_t.t(), out_dtype=torch.float32, out=out)
                self._mm_f32_out = True
                return
            except (TypeError, RuntimeError):
                self._mm_f32_out = False
        if self._mm_f32_out:
            torch.mm(a, b_t.t(), out_dtype=torch.float32, out=out)
        else:
            out.copy_(torch.mm(a, b_t.t(), out_dtype=torch.float32))

    # ------------------------------------------------------------------------------------------
    def _attend(self, i, a: LegavikAttention, qf, gate, out, out_scale, meta: BatchMeta, T):
        """Softmax attention of the step's queries over the layer's cache rows, one sigmoid gate per head, into `out` [T, H, DV]."""
        attend_window(qf, self.cache_k[i], self.cache_v[i], out, meta, a.window or FULL_WINDOW, a.scale, tiles=self.use_tiles,
                      min_tokens=self.tiles_min_tokens, min_ctas=self.prompt_tiles_min_ctas, gate=gate, gate_per_head=True,
                      keep_first=a.keep_first if a.window else 0, out_scale=out_scale)

    def _attention(self, i, m, p, h, meta, T):
        a = m.att
        H, G, D, DV = a.heads, a.kv_heads, a.dim, a.vdim
        ld = (H + G) * D + H
        proj = self.buf_proj[:T * ld].view(T, ld)
        torch.matmul(h, p.w_in.t(), out=proj)
        qf = self.buf_q[:T * H * D].view(T, H, D)
        ops.seq_head_prep(proj, 0, H * D, None, qf, self.cache_k[i], self.cache_v[i], meta.table, H, self.cfg.eps, norm_last=True,
                          inv_freq=p.inv_freq, rot_dims=a.rot_dims, rot_amp=p.rot_amp, keep_first=a.keep_first if a.window else 0)
        att = self.buf_att[:T * H * DV].view(T, H, DV)
        self._attend(i, a, qf, proj[:, (H + G) * D:], att, 1.0, meta, T)
        return att.view(T, H * DV), None

    def _parallel(self, i, m, p, h, meta, T):
        a, dl, eps = m.att, m.delta, self.cfg.eps
        H, G, D, DV = a.heads, a.kv_heads, a.dim, a.vdim
        ld = p.w_in.shape[0]
        proj = self.buf_proj[:T * ld].view(T, ld)
        torch.addmm(p.b_in, h, p.w_in.t(), out=proj)                                             # the left half's biases, zeros elsewhere
        left = (H + G) * D + G * DV                                                              # columns of the left q, k, v
        right = 2 * dl.kv_heads * dl.dim + dl.heads * dl.vdim                                    # columns of the right q, k, v
        at_a1 = left + right
        at_g1 = at_a1 + dl.decay_rank
        at_gate = at_g1 + dl.gate_rank
        at_beta = at_gate + H
        wide = H * DV + dl.heads * dl.vdim
        att = self.buf_att[:T * wide].view(T, wide)
        # right half: decays and output gates from their two-stage projections, then everything else in the delta rule's kernels
        decay = self.buf_decay[:T * dl.heads * dl.dim].view(T, dl.heads * dl.dim)
        self._mm_to_f32(proj[:, at_a1:at_g1], p.a2, decay)                                       # what enters an exponential stays float32
        gate = self.buf_gate[:T * dl.heads * dl.vdim].view(T, dl.heads * dl.vdim)
        torch.mm(proj[:, at_g1:at_gate], p.g2.t(), out=gate)
        ops.seq_delta_channel(proj[:, left:], at_beta - left, p.conv_r, self.tail_r[i], decay, p.A_log, p.dt_bias, p.r_norm, gate,
                              self.rec_state[i], att[:, H * DV:], meta, dl.kv_heads, eps, scratch=self.scan_scratch, unit_eps=UNIT_EPS,
                              out_scale=m.right_scale)
        # left half
        qf = self.buf_q[:T * H * D].view(T, H, D)
        ops.seq_head_prep(proj, 0, H * D, (H + G) * D, qf, self.cache_k[i], self.cache_v[i], meta.table, H, eps, conv_w=p.conv_l,
                          tail=self.tail_l[i], qn_w=p.q_norm, kn_w=p.k_norm, inv_freq=p.inv_freq, rot_dims=a.rot_dims, rot_amp=p.rot_amp,
                          temp_coef=a.temp_coef, temp_every=a.temp_every, keep_first=a.keep_first if a.window else 0)
        self._attend(i, a, qf, proj[:, at_gate:at_beta], att.as_strided((T, H, DV), (wide, DV, 1)), m.left_scale, meta, T)
        return att, p.o_b

    @torch.no_grad()
    def forward_batch(self, input_ids: torch.Tensor, meta: BatchMeta, trace: Optional[list] = None) -> torch.Tensor:
        """input_ids: int32 [ntok] on the device. Returns the final-norm hidden state [ntok, W] (activation type), a view of
        the arena. `trace`, if a list, receives a copy of the residual stream after every layer (debugging)."""
        cfg, T, W = self.cfg, meta.ntok, self.cfg.width
        if T > self.max_step_tokens or input_ids.numel() != T:
            raise ValueError(f"forward_batch: {T} tokens (at most {self.max_step_tokens})")
        x = self.buf_x[:T * W].view(T, W)
        h = self.buf_h[:T * W].view(T, W)
        y = self.buf_y[:T * W].view(T, W)
        ops.seq_embed(self.embed, input_ids, x)
        n = len(cfg.layers)
        first = self.weights[0].norm1 if n else self.final_norm
        ops.seq_residual_tanh(x, first.alpha, first.w, first.b, out=h)
        for i in range(n):
            p, m, f = self.weights[i], cfg.layers[i].mixer, cfg.layers[i].mlp
            after = self.weights[i + 1].norm1 if i + 1 < n else self.final_norm                 # the norm that reads this layer's result
            mid = p.norm2 if f is not None else after
            att, bias = (self._attention if m.kind == "attention" else self._parallel)(i, m, p, h, meta, T)
            torch.matmul(att, p.o.t(), out=y)
            ops.seq_residual_tanh(x, mid.alpha, mid.w, mid.b, y=y, y_bias=bias, x_out=x, out=h)
            if f is not None:
                idx = self.buf_idx[:T * f.top].view(T, f.top)
                rw = self.buf_rw[:T * f.top].view(T, f.top)
                pair = self.buf_pair[:T * f.top * W].view(T, f.top, W)
                ops.moe_route_grouped(h, p.router, None, idx, rw, score="softmax", groups=f.groups, keep=f.keep, group_top=GROUP_TOP,
                                      normalize=True)
                run_experts(h, p.gate_up, p.edown, idx, pair, f.experts, f.ff, tiles=self.use_tiles)
                ops.seq_residual_tanh(x, after.alpha, after.w, after.b, y=pair, y_w=rw, x_out=x, out=h)
            if trace is not None:
                trace.append(x.clone())
        return h

    @torch.no_grad()
    def logits(self, hidden_rows: torch.Tensor) -> torch.Tensor:
        """float32 logits [n, vocab] of final-norm hidden rows [n, W], soft-capped."""
        if self.dtype == torch.float32:
            out = torch.matmul(hidden_rows, self.head.t())
        else:
            out = torch.mm(hidden_rows, self.head.t(), out_dtype=torch.float32)
        if self.cfg.logit_softcap:
            ops.seq_softcap(out, self.cfg.logit_softcap)
        return out
