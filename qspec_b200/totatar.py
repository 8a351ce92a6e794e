"""Totatar: a decoder with a norm before and after every sublayer that mixes Mamba-2 layers with layers that run sliding-window attention
with a sink and scalar-decay linear attention side by side, followed by dense or routed feed-forward layers.

With x the float32 residual stream and N(v; g) = v / sqrt(mean(v^2) + eps) * (1 + g):

    x = embed[token]
    x <- x + N(mixer(N(x; norm1)); norm1b);      x <- x + N(ff(N(x; norm2)); norm2b)          (a layer may have no feed-forward)
    logits = embed N(x; final.norm)                                                            (the embedding table is the output matrix)

mixers (`layers[i].type`):
    parallel    left_scale * left + right_scale * right of the same h:
      left      q, k, v with biases; the first `rot.dims` entries of every q and k head rotated (entry 2i with 2i + 1, frequencies divided
                by `rot.scaling.factor`); position i sees j when 0 <= i - j < mask.size; the softmax denominator carries exp(sink_head);
                W_o.
      right     q, k, v = silu(W h); per head S <- decay S + k v^T, o = S^T q; all heads normed together, times a plain weight and
                sigmoid(W_g h); W_o.
    mamba2      [z | x | B | C | dt] = W_in h; x, B, C through a short causal convolution with bias and silu; dt = softplus(dt + dt_bias);
                per head (heads / groups of them share B and C) S <- exp(-exp(A_log) dt) S + dt B x^T, y = S^T C + D x; y * silu(z) normed
                in norm_groups equal parts, times a plain weight; W_o.
feed-forward (`mlp.kind`):
    dense       W_down (gelu_tanh(W_gate h) * W_up h)
    moe         logits W_router h + bias in float32; the `top` largest, weighted by a softmax over those alone; expert(h) = W_down
                (silu(W_gate h) * W_up h); a shared expert of the same form runs for every token.

Wiring follows `legavik.LegavikModel`: a flat token batch with per-token slot and position (`state.BatchMeta`), state held by the model
and indexed by slot, a scratch arena allocated once, dense products in the vendor library, everything else in the sequence-mixer kernel
library (`ops.seq_*`, `ops.moe_*`). One product makes everything a mixer reads from h, one product closes it (the two halves of a
parallel layer write side by side, already scaled). Every residual sum sits between the norm of a sublayer's result and the norm of the
next one's input in one launch (`ops.seq_sandwich_norm`). Both recurrences run through `ops.seq_scalar_decay`. Per-slot state: key / value
rings of the attention, the float32 matrices of both recurrences, and the last `conv - 1` inputs of every convolution (double-buffered by
the step's phase). Nothing is cleared when a slot is released: cache rows are valid by position, the recurrences start from zero at
position 0.
"""
from __future__ import annotations

import json
import math
import os
from dataclasses import dataclass, field
from typing import Dict, List, Optional, Tuple

import torch

from . import ops
from .seq_layers import PROMPT_TILES_MIN_CTAS, TILES_MIN_TOKENS, attend_window, run_experts
from .state import CHUNK_MIN, BatchMeta

FULL_WINDOW = 1 << 30               # attention over the whole sequence: a window no sequence reaches
SECTION = 8                         # sections of a fused row start on multiples of this many entries (16 bytes of bfloat16)
NO_DECAY_LOG = -1e30                # stands for the logarithm of a decay of zero


@dataclass
class TotatarAttention:
    """The left half of a parallel mixer."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int] = None    # None: the whole sequence
    rot_dims: int = 0
    rot_base: float = 10000.0
    rot_factor: float = 1.0


@dataclass
class TotatarLinear:
    """The right half of a parallel mixer."""
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...] = ()


@dataclass
class TotatarMamba2:
    heads: int
    groups: int
    state: int
    vdim: int
    conv: int
    norm_groups: int = 1

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:      # of the convolution
        return self.inner + 2 * self.groups * self.state


@dataclass
class TotatarMixer:
    kind: str                       # "parallel" | "mamba2"
    att: Optional[TotatarAttention] = None
    lin: Optional[TotatarLinear] = None
    ssm: Optional[TotatarMamba2] = None
    left_scale: float = 1.0
    right_scale: float = 1.0


@dataclass
class TotatarFF:
    kind: str                       # "dense" | "moe"
    ff: int                         # hidden size (of one expert for "moe")
    experts: int = 0
    top: int = 0
    shared_ff: int = 0              # 0: no shared expert


@dataclass
class TotatarLayer:
    mixer: TotatarMixer
    mlp: Optional[TotatarFF]


def _attention_from(m: dict, i: int) -> TotatarAttention:
    rot, mask = m.get("rot") or {}, m.get("mask") or {}
    heads, dim = int(m["heads"]), int(m["dim"])
    a = TotatarAttention(heads=heads, kv_heads=int(m.get("kv_heads", heads)), dim=dim, vdim=int(m.get("vdim", dim)), scale=float(m["scale"]),
                         window=int(mask["size"]) if mask.get("size") else None, rot_dims=int(rot.get("dims", 0)),
                         rot_base=float(rot.get("base", 10000.0)), rot_factor=float((rot.get("scaling") or {}).get("factor", 1.0)))
    if a.kv_heads < 1 or a.heads % a.kv_heads:
        raise ValueError(f"layer {i}: {a.heads} heads over {a.kv_heads} key heads")
    if a.rot_dims % 2 or not 0 <= a.rot_dims <= a.dim:
        raise ValueError(f"layer {i}: {a.rot_dims} rotated dimensions of {a.dim}")
    if (a.window is not None and a.window < 1) or a.rot_factor <= 0:
        raise ValueError(f"layer {i}: a window of {a.window}, a rotation stretched by {a.rot_factor}")
    return a


@dataclass
class TotatarConfig:
    vocab: int
    width: int
    eps: float
    layers: List[TotatarLayer] = field(default_factory=list)
    name: str = "totatar"

    @staticmethod
    def from_dict(d: dict) -> "TotatarConfig":
        layers = []
        for i, e in enumerate(d["layers"]):
            kind, m = e.get("type"), e["mixer"]
            if kind == "parallel":
                r = m["right"]
                lin = TotatarLinear(heads=int(r["heads"]), dim=int(r["dim"]), vdim=int(r.get("vdim", r["dim"])),
                                    decay=tuple(float(v) for v in r["decay"]))
                if len(lin.decay) != lin.heads or any(not 0.0 <= v <= 1.0 for v in lin.decay):
                    raise ValueError(f"layer {i}: {lin.heads} heads need as many decays between 0 and 1, not {list(lin.decay)}")
                mixer = TotatarMixer(kind=kind, att=_attention_from(m["left"], i), lin=lin, left_scale=float(m.get("left_scale", 1.0)),
                                     right_scale=float(m.get("right_scale", 1.0)))
            elif kind == "mamba2":
                s = TotatarMamba2(heads=int(m["heads"]), groups=int(m.get("groups", 1)), state=int(m["state"]), vdim=int(m["vdim"]),
                                  conv=int(m["conv"]), norm_groups=int(m.get("norm_groups", 1)))
                if s.groups < 1 or s.heads % s.groups or s.conv < 1 or s.norm_groups < 1 or s.inner % s.norm_groups:
                    raise ValueError(f"layer {i}: {s.heads} heads in {s.groups} groups, a convolution of {s.conv} taps, {s.inner} channels in "
                                     f"{s.norm_groups} norm groups")
                mixer = TotatarMixer(kind=kind, ssm=s)
            else:
                raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
            f = e.get("mlp")
            if f is None:
                mlp = None
            elif f.get("kind") == "dense":
                mlp = TotatarFF(kind="dense", ff=int(f["ff"]))
            elif f.get("kind") == "moe":
                r = f["router"]
                mlp = TotatarFF(kind="moe", ff=int(f["expert"]["ff"]), experts=int(r["experts"]), top=int(r["top"]),
                                shared_ff=int((f.get("shared") or {}).get("ff", 0)))
                if not 1 <= mlp.top <= mlp.experts:
                    raise ValueError(f"layer {i}: top {mlp.top} of {mlp.experts} experts")
            else:
                raise ValueError(f"layer {i}: unknown feed-forward kind {f.get('kind')!r}")
            layers.append(TotatarLayer(mixer=mixer, mlp=mlp))
        return TotatarConfig(vocab=int(d["vocab"]), width=int(d["width"]), eps=float(d["norm"]["eps"]), layers=layers)

    def to_dict(self) -> dict:
        out = {"architecture": "Totatar", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps}, "layers": []}
        for l in self.layers:
            m, f = l.mixer, l.mlp
            if m.kind == "parallel":
                a, r = m.att, m.lin
                left = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale}
                if a.window is not None:
                    left["mask"] = {"size": a.window}
                if a.rot_dims:
                    left["rot"] = {"base": a.rot_base, "dims": a.rot_dims, "scaling": {"factor": a.rot_factor}}
                mx = {"left": left, "right": {"heads": r.heads, "dim": r.dim, "vdim": r.vdim, "decay": list(r.decay)},
                      "left_scale": m.left_scale, "right_scale": m.right_scale}
            else:
                s = m.ssm
                mx = {"heads": s.heads, "groups": s.groups, "state": s.state, "vdim": s.vdim, "conv": s.conv, "norm_groups": s.norm_groups}
            if f is None:
                mlp = None
            elif f.kind == "dense":
                mlp = {"kind": "dense", "ff": f.ff}
            else:
                mlp = {"kind": "moe", "expert": {"ff": f.ff}, "router": {"experts": f.experts, "top": f.top},
                       "shared": {"ff": f.shared_ff} if f.shared_ff else None}
            out["layers"].append({"type": m.kind, "mixer": mx, "mlp": mlp})
        return out

    def tensor_shapes(self) -> Dict[str, tuple]:
        """Name -> shape of every tensor a checkpoint of this configuration must hold."""
        W = self.width
        out = {"embed": (self.vocab, W)}

        def ff(y, hidden):
            out.update({y + "gate": (hidden, W), y + "up": (hidden, W), y + "down": (W, hidden)})

        for i, l in enumerate(self.layers):
            m, f, p = l.mixer, l.mlp, f"l{i}."
            out.update({p + "norm1": (W,), p + "norm1b": (W,)})
            x = p + "mix."
            if m.kind == "parallel":
                a, r, y = m.att, m.lin, x + "left."
                for n, rows in (("q", a.heads * a.dim), ("k", a.kv_heads * a.dim), ("v", a.kv_heads * a.vdim)):
                    out.update({y + n: (rows, W), y + n + ".b": (rows,)})
                out.update({y + "sink": (a.heads,), y + "o": (W, a.heads * a.vdim)})
                y = x + "right."
                out.update({y + "q": (r.heads * r.dim, W), y + "k": (r.heads * r.dim, W), y + "v": (r.heads * r.vdim, W),
                            y + "g": (r.heads * r.vdim, W), y + "norm": (r.heads * r.vdim,), y + "o": (W, r.heads * r.vdim)})
            else:
                s = m.ssm
                out.update({x + "in": (s.inner + s.channels + s.heads, W), x + "conv": (s.channels, s.conv), x + "conv.b": (s.channels,),
                            x + "dt_bias": (s.heads,), x + "A_log": (s.heads,), x + "D": (s.heads,), x + "norm": (s.inner,),
                            x + "o": (W, s.inner)})
            if f is None:
                continue
            out.update({p + "norm2": (W,), p + "norm2b": (W,)})
            y = p + "mlp."
            if f.kind == "dense":
                ff(y, f.ff)
            else:
                for e in range(f.experts):
                    ff(y + f"e{e}.", f.ff)
                out.update({y + "router": (f.experts, W), y + "router.b": (f.experts,)})
                if f.shared_ff:
                    ff(y + "shared.", f.shared_ff)
        out["final.norm"] = (W,)
        return out


def random_weights(cfg: TotatarConfig, seed: int = 0) -> Dict[str, torch.Tensor]:
    """Random bfloat16 tensors of a configuration (CPU): matrices ~ N(0, 1/fan_in), norm weights small around zero (plain ones around
    one), Mamba-2 rates and step sizes in the range where the state neither dies nor saturates."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in cfg.tensor_shapes().items():
        if name.endswith(".A_log"):
            t = torch.log(1.0 + 7.0 * torch.rand(shape, generator=g))
        elif name.endswith(".dt_bias"):
            t = -2.5 + torch.randn(shape, generator=g)
        elif name.endswith((".D", "right.norm", "mix.norm")):
            t = 1.0 + 0.1 * torch.randn(shape, generator=g)
        elif name.endswith(".conv"):
            t = torch.randn(shape, generator=g) / shape[1] ** 0.5
        elif name.endswith(".sink"):
            t = torch.randn(shape, generator=g)
        elif len(shape) == 2:
            t = torch.randn(shape, generator=g) / shape[1] ** 0.5
        else:
            t = 0.1 * torch.randn(shape, generator=g)
        out[name] = t.to(torch.bfloat16)
    return out


def _sections(sizes) -> Tuple[List[int], int]:
    """First entries of sections laid one after the other on SECTION boundaries, and the length of the whole row."""
    offs, at = [], 0
    for n in sizes:
        offs.append(at)
        at += -(-n // SECTION) * SECTION
    return offs, at


class _LayerWeights:
    """Device tensors of one layer: large matrices in the activation type (everything that reads the mixer's input in one, the output
    matrices of a parallel layer side by side), vectors, convolutions, the router and everything a recurrence reads in float32."""

    def __init__(self, cfg: TotatarConfig, i: int, sd: Dict[str, torch.Tensor], dtype, device):
        spec, p = cfg.layers[i], f"l{i}."
        m, f = spec.mixer, spec.mlp

        def laid(parts, dim=0):
            """Tensors joined along `dim`, each starting on a section boundary (zeros between). Returns the tensor and the starts."""
            offs, total = _sections([t.shape[dim] for t in parts])
            shape = list(parts[0].shape)
            shape[dim] = total
            out = torch.zeros(shape, dtype=parts[0].dtype)
            for t, o in zip(parts, offs):
                out.narrow(dim, o, t.shape[dim]).copy_(t)
            return out, offs

        big = lambda t: t.to(device=device, dtype=dtype).contiguous()
        small = lambda t: t.to(device=device, dtype=torch.float32).contiguous()
        norm = lambda name: small(sd[p + name])
        self.norm1, self.norm1b = norm("norm1"), norm("norm1b")
        if m.kind == "parallel":
            a, r = m.att, m.lin
            L, R = p + "mix.left.", p + "mix.right."
            w, (self.q, self.k, self.v, self.rq, self.rk, self.rv, self.rg) = laid([sd[L + n] for n in "qkv"] + [sd[R + n] for n in "qkvg"])
            self.w_in = big(w)
            bias = torch.zeros(w.shape[0], dtype=torch.float32)
            for n, o in (("q", self.q), ("k", self.k), ("v", self.v)):
                b = sd[L + n + ".b"].to(torch.float32)
                bias[o:o + b.numel()] = b
            self.b_in = big(bias)
            o, (_, self.o_right) = laid([sd[L + "o"], sd[R + "o"]], dim=1)                     # columns [left heads | right heads]
            self.o = big(o)
            self.sink = small(sd[L + "sink"])
            self.inv_freq = None
            if a.rot_dims:
                i2 = torch.arange(a.rot_dims // 2, dtype=torch.float64)
                self.inv_freq = small(torch.tensor(a.rot_base, dtype=torch.float64) ** (-2.0 * i2 / a.rot_dims) / a.rot_factor)
            self.r_norm = small(sd[R + "norm"])
            self.decay = small(torch.tensor(r.decay, dtype=torch.float64))
            self.log_decay = small(torch.tensor([math.log(v) if v > 0.0 else NO_DECAY_LOG for v in r.decay], dtype=torch.float64))
        else:
            s, x = m.ssm, p + "mix."
            gn = s.groups * s.state
            z, xs, B, C, dt = torch.split(sd[x + "in"], [s.inner, s.inner, gn, gn, s.heads], dim=0)
            w, (self.z, self.x, self.B, self.C, self.dt) = laid([z, xs, B, C, dt])
            self.w_in = big(w)
            self.conv = small(laid(list(torch.split(sd[x + "conv"], [s.inner, gn, gn], dim=0)))[0])       # channel = column - self.x
            self.conv_b = small(laid(list(torch.split(sd[x + "conv.b"], [s.inner, gn, gn], dim=0)))[0])
            self.dt_bias, self.A_log, self.D = (small(sd[x + n]) for n in ("dt_bias", "A_log", "D"))
            self.m_norm = small(sd[x + "norm"])
            self.o = big(sd[x + "o"])
        if f is None:
            return
        self.norm2, self.norm2b = norm("norm2"), norm("norm2b")
        y = p + "mlp."
        if f.kind == "dense":
            self.gate_up, self.down = big(torch.cat([sd[y + "gate"], sd[y + "up"]], 0)), big(sd[y + "down"])
        else:
            self.router, self.router_b = small(sd[y + "router"]), small(sd[y + "router.b"])
            self.egate_up = big(torch.stack([torch.cat([sd[y + f"e{e}.gate"], sd[y + f"e{e}.up"]], 0) for e in range(f.experts)]))
            self.edown = big(torch.stack([sd[y + f"e{e}.down"] for e in range(f.experts)]))
            if f.shared_ff:
                self.gate_up, self.down = big(torch.cat([sd[y + "shared.gate"], sd[y + "shared.up"]], 0)), big(sd[y + "shared.down"])


class TotatarModel(torch.nn.Module):
    """Weights, per-slot state and the forward pass over a flat token batch (`state.BatchMeta`).

    dtype: torch.bfloat16 (serving: bfloat16 matrix products with float32 accumulation) or torch.float32 (everything in true
    float32). n_slots sequences can be live at once; a step carries at most max_step_tokens tokens. Window layers keep a ring of window -
    1 + max_step_tokens rows per slot, so that a sequence may be of any length; where a layer attends over all of it, it holds at most
    max_seq_tokens tokens."""

    architecture = "Totatar"
    DEFAULT_SEQ_TOKENS = 8192

    def __init__(self, cfg: TotatarConfig, weights: Dict[str, torch.Tensor], dtype=torch.bfloat16, device="cuda",
                 n_slots: int = 8, max_step_tokens: int = 2048, max_seq_tokens: Optional[int] = None):
        super().__init__()
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("TotatarModel: dtype must be torch.bfloat16 or torch.float32")
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
        self.final_norm = weights["final.norm"].to(**f32).contiguous()
        self.weights = [_LayerWeights(cfg, i, weights, dtype, dev) for i in range(len(cfg.layers))]
        # ---- per-slot state ----
        limit = max(int(max_seq_tokens or self.DEFAULT_SEQ_TOKENS), 1)
        bounded = False                                                                        # whether a cache bounds the sequence length
        self.cache_k: Dict[int, torch.Tensor] = {}                                             # layer -> [slots, rows, G, D]
        self.cache_v: Dict[int, torch.Tensor] = {}                                             # layer -> [slots, rows, G, DV]
        self.rec_state: Dict[int, torch.Tensor] = {}                                           # layer -> float32 [slots, H, D, DV]
        self.tail: Dict[int, torch.Tensor] = {}                                                # layer -> float32 [2, slots, taps - 1, C]
        for i, l in enumerate(cfg.layers):
            m = l.mixer
            if m.kind == "parallel":
                a, r = m.att, m.lin
                rows = limit if a.window is None else min(a.window - 1 + T, limit)
                bounded |= a.window is None or rows < a.window - 1 + T
                self.cache_k[i] = torch.zeros(n_slots, rows, a.kv_heads, a.dim, **act)
                self.cache_v[i] = torch.zeros(n_slots, rows, a.kv_heads, a.vdim, **act)
                self.rec_state[i] = torch.zeros(n_slots, r.heads, r.dim, r.vdim, **f32)
            else:
                s = m.ssm
                self.tail[i] = torch.zeros(2, n_slots, s.conv - 1, self.weights[i].conv.shape[0], **f32)
                self.rec_state[i] = torch.zeros(n_slots, s.heads, s.state, s.vdim, **f32)
        self.max_seq_len = limit if bounded else None                                          # checked by the scheduler
        # ---- scratch arena, allocated once ----
        mx = lambda vals: max(list(vals) + [1])
        mix = [l.mixer for l in cfg.layers]
        ffs = [l.mlp for l in cfg.layers if l.mlp]
        moe = [f for f in ffs if f.kind == "moe"]
        hidden = [f.ff if f.kind == "dense" else f.shared_ff for f in ffs]
        self.buf_x = torch.empty(T * W, **f32)                                                 # residual stream (updated in place)
        self.buf_h = torch.empty(T * W, **act)                                                 # sublayer input
        self.buf_y = torch.empty(T * W, **act)                                                 # sublayer output
        self.buf_proj = torch.empty(T * mx(w.w_in.shape[0] for w in self.weights), **act)
        self.buf_q = torch.empty(T * mx(m.att.heads * m.att.dim for m in mix if m.att), **f32)               # rotated queries
        self.buf_rec = torch.empty(T * mx(t.shape[1] * t.shape[3] for t in self.rec_state.values()), **f32)  # read-outs of a recurrence
        self.buf_conv = torch.empty(T * mx(t.shape[3] for t in self.tail.values()), **act)
        self.buf_att = torch.zeros(T * mx(w.o.shape[1] for w in self.weights), **act)          # what W_o reads (finite between the sections)
        self.buf_gu = torch.empty(T * 2 * mx(hidden), **act)
        self.buf_ff = torch.empty(T * mx(hidden), **act)
        chunks = max(T // CHUNK_MIN, 1)                                                        # ceil(n / 64) <= n / 32 for every segment that has chunks
        self.scan_scratch = torch.empty(mx(ops.seq_scalar_decay_scratch_bytes(chunks, *t.shape[1:]) for t in self.rec_state.values())
                                        if dtype == torch.bfloat16 else 16, dtype=torch.uint8, device=dev)
        tops = mx(f.top for f in moe)
        self.buf_idx = torch.empty(T * tops, dtype=torch.int32, device=dev)
        self.buf_rw = torch.empty(T * tops, **f32)
        self.buf_pair = torch.empty(T * tops * W if moe else 1, **act)
        # bfloat16 takes the tensor-core forms where the sizes allow; QSPEC_SEQ_TILES=0 keeps the plain ones
        self.use_tiles = dtype == torch.bfloat16 and os.environ.get("QSPEC_SEQ_TILES", "1") != "0"
        self.tiles_min_tokens, self.prompt_tiles_min_ctas = TILES_MIN_TOKENS, PROMPT_TILES_MIN_CTAS

    # ------------------------------------------------------------------------------------------
    @classmethod
    def from_pretrained(cls, path: str, dtype=torch.bfloat16, device="cuda", **kw) -> "TotatarModel":
        from .checkpoint import read_safetensors_file
        with open(os.path.join(path, "config.json")) as f:
            cfg = TotatarConfig.from_dict(json.load(f))
        return cls(cfg, read_safetensors_file(os.path.join(path, "model.safetensors")), dtype=dtype, device=device, **kw)

    @property
    def vocab_size(self) -> int:
        return self.cfg.vocab

    def state_bytes_per_slot(self) -> int:
        ts = [t for d in (self.cache_k, self.cache_v, self.rec_state, self.tail) for t in d.values()]
        return sum(t.numel() * t.element_size() // self.n_slots for t in ts)

    # ------------------------------------------------------------------------------------------
    def _parallel(self, i, m, p, h, meta, T):
        a, r, eps = m.att, m.lin, self.cfg.eps
        H, D, DV = a.heads, a.dim, a.vdim
        ld, wide, rv = p.w_in.shape[0], p.o.shape[1], r.heads * r.vdim
        proj = self.buf_proj[:T * ld].view(T, ld)
        torch.addmm(p.b_in, h, p.w_in.t(), out=proj)                                             # the left half's biases, zeros elsewhere
        att = self.buf_att[:T * wide].view(T, wide)
        # right half: linear attention, all heads normed together
        rec = self.buf_rec[:T * rv].view(T, rv)
        ops.seq_scalar_decay(proj, p.rq, p.rk, p.rv, r.heads, self.rec_state[i], rec, meta, decay=p.decay, log_decay=p.log_decay,
                             scratch=self.scan_scratch if self.use_tiles else None)
        ops.seq_part_norm(rec, p.r_norm, proj[:, p.rg:p.rg + rv], "sigmoid_after", att[:, p.o_right:p.o_right + rv], eps,
                          out_scale=m.right_scale)
        # left half: window attention with a sink
        qf = self.buf_q[:T * H * D].view(T, H, D)
        ops.seq_head_prep(proj, p.q, p.k, p.v, qf, self.cache_k[i], self.cache_v[i], meta.table, H, eps, norm=False, inv_freq=p.inv_freq,
                          rot_dims=a.rot_dims, pairing="interleaved")
        attend_window(qf, self.cache_k[i], self.cache_v[i], att.as_strided((T, H, DV), (wide, DV, 1)), meta, a.window or FULL_WINDOW,
                      a.scale, tiles=self.use_tiles, min_tokens=self.tiles_min_tokens, min_ctas=self.prompt_tiles_min_ctas, sink=p.sink,
                      out_scale=m.left_scale)
        return att

    def _mamba2(self, i, m, p, h, meta, T):
        s = m.ssm
        ld, C, inner = p.w_in.shape[0], p.conv.shape[0], s.inner
        proj = self.buf_proj[:T * ld].view(T, ld)
        torch.matmul(h, p.w_in.t(), out=proj)
        rec = self.buf_rec[:T * inner].view(T, inner)
        ops.seq_scalar_decay(proj, p.C, p.B, p.x, s.groups, self.rec_state[i], rec, meta, dt=proj[:, p.dt:p.dt + s.heads], dt_bias=p.dt_bias,
                             A_log=p.A_log, D_skip=p.D, conv=(p.conv, p.conv_b, p.x, self.tail[i]),
                             conv_out=self.buf_conv[:T * C].view(T, C), scratch=self.scan_scratch if self.use_tiles else None)
        att = self.buf_att[:T * inner].view(T, inner)
        ops.seq_part_norm(rec, p.m_norm, proj[:, p.z:p.z + inner], "silu_before", att, self.cfg.eps, parts=s.norm_groups)
        return att

    def _glu(self, p, h, hidden, act, out, T):
        """down(act(gate h) * up h): a dense feed-forward layer, or the shared expert."""
        gu = self.buf_gu[:T * 2 * hidden].view(T, 2 * hidden)
        torch.matmul(h, p.gate_up.t(), out=gu)
        ff = self.buf_ff[:T * hidden].view(T, hidden)
        ops.seq_glu(gu, ff, act)
        torch.matmul(ff, p.down.t(), out=out)

    @torch.no_grad()
    def forward_batch(self, input_ids: torch.Tensor, meta: BatchMeta, trace: Optional[list] = None) -> torch.Tensor:
        """input_ids: int32 [ntok] on the device. Returns the final-norm hidden state [ntok, W] (activation type), a view of
        the arena. `trace`, if a list, receives a copy of the residual stream after every layer (debugging)."""
        cfg, T, W, eps = self.cfg, meta.ntok, self.cfg.width, self.cfg.eps
        if T > self.max_step_tokens or input_ids.numel() != T:
            raise ValueError(f"forward_batch: {T} tokens (at most {self.max_step_tokens})")
        x = self.buf_x[:T * W].view(T, W)
        h = self.buf_h[:T * W].view(T, W)
        y = self.buf_y[:T * W].view(T, W)
        ops.seq_embed(self.embed, input_ids, x)
        n = len(cfg.layers)
        ops.seq_sandwich_norm(x, eps, pre_w=self.weights[0].norm1 if n else self.final_norm, out=h)
        for i in range(n):
            p, m, f = self.weights[i], cfg.layers[i].mixer, cfg.layers[i].mlp
            after = self.weights[i + 1].norm1 if i + 1 < n else self.final_norm                 # the norm that reads this layer's result
            att = (self._parallel if m.kind == "parallel" else self._mamba2)(i, m, p, h, meta, T)
            torch.matmul(att, p.o.t(), out=y)
            ops.seq_sandwich_norm(x, eps, y=y, post_w=p.norm1b, pre_w=p.norm2 if f is not None else after, x_out=x, out=h)
            if f is not None and f.kind == "dense":
                self._glu(p, h, f.ff, "gelu_tanh", y, T)
                ops.seq_sandwich_norm(x, eps, y=y, post_w=p.norm2b, pre_w=after, x_out=x, out=h)
            elif f is not None:
                idx = self.buf_idx[:T * f.top].view(T, f.top)
                rw = self.buf_rw[:T * f.top].view(T, f.top)
                pair = self.buf_pair[:T * f.top * W].view(T, f.top, W)
                ops.moe_route_chosen(h, p.router, idx, rw, bias=p.router_b)
                run_experts(h, p.egate_up, p.edown, idx, pair, f.experts, f.ff, tiles=self.use_tiles)
                if f.shared_ff:
                    self._glu(p, h, f.shared_ff, "silu", y, T)
                ops.seq_sandwich_norm(x, eps, y=pair, y_w=rw, y2=y if f.shared_ff else None, post_w=p.norm2b, pre_w=after, x_out=x, out=h)
            if trace is not None:
                trace.append(x.clone())
        return h

    @torch.no_grad()
    def logits(self, hidden_rows: torch.Tensor) -> torch.Tensor:
        """float32 logits [n, vocab] of final-norm hidden rows [n, W]; the embedding table is the output matrix."""
        if self.dtype == torch.float32:
            return torch.matmul(hidden_rows, self.embed.t())
        return torch.mm(hidden_rows, self.embed.t(), out_dtype=torch.float32)
