"""Plain implementation of the Legavik design: float64, whole sequences, no cache, one function per mechanism.

It shares no code with the product path (`qspec_b200/legavik.py` and its kernels) and is the reference of the tests.
`cfg` is the dictionary of a config.json, `w` maps tensor names to torch tensors (any float type; read as float64).

    norm:       T(x; n) = tanh(n.alpha * x) * n + n.b, nothing is averaged
    layer:      x <- x + mixer(T(x; norm1));   x <- x + ff(T(x; norm2))
    attention:  q = W_q h, k = W_k h, v = k; q, k rotated with stretched frequencies and an amplitude, then unit_rms per head; softmax over
                the last `size` positions and the first `keep_first` ones; head * sigmoid(W_g h)_head; W_o
    parallel:   left_scale * L(h) + right_scale * R(h)
      L         q, k, v = conv(W h + b); q, k = unit_rms * weight; q * (1 + coef ln(floor((p + 1) / every) + 1)); causal softmax;
                head * sigmoid(W_g h)_head; W_o + bias
      R         q, k, v = silu(conv(W h)); q, k unit vectors (q / sqrt(dim)); per head and key channel
                g = exp(-exp(A_log) softplus(W_a2 W_a1 h + dt_bias)); S <- diag(g) S; u = sigmoid(W_b h) (v - S^T k); S <- S + k u^T;
                o = S^T q; W_o (unit_rms(o) * norm * sigmoid(W_g2 W_g1 h))
    ff:         s = softmax(W_r h); the best groups by their largest score; the largest scores in them, divided by their sum;
                sum of weight * W_down (silu(W_gate h) * W_up h)
    end:        logits = cap tanh(head T(x; final.norm) / cap)
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64


def _t(w: Dict[str, torch.Tensor], name: str) -> torch.Tensor:
    return w[name].to(F64)


def tanh_norm(x: torch.Tensor, w, name: str) -> torch.Tensor:
    return torch.tanh(_t(w, name + ".alpha") * x) * _t(w, name) + _t(w, name + ".b")


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.where(z > 30.0, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


def causal_conv(x: torch.Tensor, taps_w: torch.Tensor) -> torch.Tensor:
    """x [T, C], taps_w [C, K]: y_t = sum_j taps_w[:, j] * x_(t - K + 1 + j), zeros before the start."""
    T, C = x.shape
    K = taps_w.shape[1]
    y = torch.zeros(T, C, dtype=F64)
    for t in range(T):
        for j in range(K):
            s = t - (K - 1) + j
            if s >= 0:
                y[t] += taps_w[:, j] * x[s]
    return y


def yarn_frequencies(dims: int, base: float, scaling: Optional[dict]) -> List[float]:
    """One frequency per rotated pair. A pair that turns more than `fast` times within `original` positions keeps its frequency,
    one that turns fewer than `slow` times is slowed down by `factor`, a ramp over the pair's index between."""
    plain = [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return plain

    def pair_of(turns):
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(pair_of(scaling["fast"])), 0)
    hi = min(math.ceil(pair_of(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / scaling["factor"] * r + f * (1.0 - r))
    return out


def yarn_amplitude(scaling: Optional[dict]) -> float:
    return 0.1 * math.log(scaling["factor"]) + 1.0 if scaling else 1.0


def rotate_halves(x: torch.Tensor, pos: torch.Tensor, freqs: List[float], amplitude: float = 1.0) -> torch.Tensor:
    """x [T, heads, n]: entry i and entry i + len(freqs) turn by pos * freqs[i] and grow by `amplitude`; the rest passes."""
    out = x.clone()
    half = len(freqs)
    for i, f in enumerate(freqs):
        a = pos.to(F64) * f
        c, s = amplitude * torch.cos(a)[:, None], amplitude * torch.sin(a)[:, None]
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * c - v * s
        out[..., i + half] = v * c + u * s
    return out


def softmax_rows(scores: torch.Tensor) -> torch.Tensor:
    e = torch.exp(scores - scores.max())
    return e / e.sum()


def masked_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, size: Optional[int] = None, keep_first: int = 0):
    """q [T, H, D], k [T, G, D], v [T, G, DV]: softmax attention of position i over the j <= i with i - j < size (None: all of
    them) or j < keep_first. Returns [T, H, DV]."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for t in range(T):
        seen = [j for j in range(t + 1) if size is None or t - j < size or j < keep_first]
        for h in range(H):
            p = softmax_rows((k[seen, h // rep] @ q[t, h]) * scale)
            out[t, h] = p @ v[seen, h // rep]
    return out


def head_gate(o: torch.Tensor, h: torch.Tensor, w, name: str) -> torch.Tensor:
    """o [T, H, DV] times one sigmoid per head."""
    return o * torch.sigmoid(h @ _t(w, name).T)[:, :, None]


def attention_mixer(h: torch.Tensor, w, p: str, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, D = m["heads"], m["kv_heads"], m["dim"]
    q = (h @ _t(w, p + "q").T).view(T, H, D)
    k = (h @ _t(w, p + "k").T).view(T, G, D)
    v = k.clone()
    rot = m.get("rot") or {}
    if rot.get("dims"):
        fr, amp = yarn_frequencies(rot["dims"], rot["base"], rot.get("scaling")), yarn_amplitude(rot.get("scaling"))
        pos = torch.arange(T)
        q, k = rotate_halves(q, pos, fr, amp), rotate_halves(k, pos, fr, amp)
    q, k = unit_rms(q, eps), unit_rms(k, eps)
    mask = m.get("mask") or {}
    o = masked_attention(q, k, v, m["scale"], mask.get("size"), mask.get("keep_first", 0))
    return head_gate(o, h, w, p + "g").reshape(T, -1) @ _t(w, p + "o").T


def temperature(pos: torch.Tensor, coef: float, every: int) -> torch.Tensor:
    return 1.0 + coef * torch.log(torch.floor((pos.to(F64) + 1.0) / every) + 1.0)


def left_mixer(h: torch.Tensor, w, p: str, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, D, DV = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (causal_conv(h @ _t(w, p + n).T + _t(w, p + n + ".b"), _t(w, p + n + ".conv")) for n in "qkv")
    q = unit_rms(q.view(T, H, D), eps) * _t(w, p + "q.norm")
    k = unit_rms(k.view(T, G, D), eps) * _t(w, p + "k.norm")
    if m.get("q_temp"):
        q = q * temperature(torch.arange(T), m["q_temp"]["coef"], m["q_temp"]["every"])[:, None, None]
    o = masked_attention(q, k, v.view(T, G, DV), m["scale"])
    return head_gate(o, h, w, p + "g").reshape(T, -1) @ _t(w, p + "o").T + _t(w, p + "o.b")


def delta_rule(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, beta: torch.Tensor, g: torch.Tensor,
               state: Optional[torch.Tensor] = None) -> torch.Tensor:
    """q, k [T, G, D] (already unit vectors), v [T, H, DV], beta [T, H], g [T, H, D]: per head every state row decays by its key
    channel's factor, the state is corrected towards v along k, and is read with q after the write. Returns o [T, H, DV];
    `state` [H, D, DV], if given, is updated in place."""
    T, H, DV = v.shape
    G, D = k.shape[1], k.shape[2]
    rep = H // G
    S = torch.zeros(H, D, DV, dtype=F64) if state is None else state
    o = torch.zeros(T, H, DV, dtype=F64)
    for t in range(T):
        for h in range(H):
            kk, qq = k[t, h // rep], q[t, h // rep]
            S[h] = g[t, h][:, None] * S[h]
            u = beta[t, h] * (v[t, h] - S[h].T @ kk)
            S[h] = S[h] + torch.outer(kk, u)
            o[t, h] = S[h].T @ qq
    return o


def right_mixer(h: torch.Tensor, w, p: str, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, D, DV = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = silu(causal_conv(h @ _t(w, p + "q").T, _t(w, p + "q.conv"))).view(T, G, D)
    k = silu(causal_conv(h @ _t(w, p + "k").T, _t(w, p + "k.conv"))).view(T, G, D)
    v = silu(causal_conv(h @ _t(w, p + "v").T, _t(w, p + "v.conv"))).view(T, H, DV)
    q = q / torch.sqrt((q * q).sum(-1, keepdim=True) + 1e-6) / math.sqrt(D)
    k = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    beta = torch.sigmoid(h @ _t(w, p + "b").T)
    a = (h @ _t(w, p + "a1").T @ _t(w, p + "a2").T + _t(w, p + "dt_bias")).view(T, H, D)
    g = torch.exp(-torch.exp(_t(w, p + "A_log"))[:, None] * softplus(a))
    o = delta_rule(q, k, v, beta, g)
    gate = torch.sigmoid(h @ _t(w, p + "g1").T @ _t(w, p + "g2").T).view(T, H, DV)
    return (unit_rms(o, eps) * _t(w, p + "norm") * gate).reshape(T, H * DV) @ _t(w, p + "o").T


def parallel_mixer(h: torch.Tensor, w, p: str, m: dict, eps: float) -> torch.Tensor:
    return m["left_scale"] * left_mixer(h, w, p + "left.", m["left"], eps) + m["right_scale"] * right_mixer(h, w, p + "right.", m["right"], eps)


def route(z: torch.Tensor, top: int, groups: int = 1, keep: int = 1):
    """One token's router logits [E] -> [(expert, weight)]."""
    s = softmax_rows(z)
    size = len(s) // groups
    best = sorted(range(groups), key=lambda gr: (-float(s[gr * size:(gr + 1) * size].max()), gr))[:keep]
    open_ = [e for e in range(len(s)) if e // size in best]
    chosen = sorted(open_, key=lambda e: (-float(s[e]), e))[:top]
    total = sum(float(s[e]) for e in chosen) + 1e-20
    return [(e, float(s[e]) / total) for e in chosen]


def expert(h: torch.Tensor, w, p: str) -> torch.Tensor:
    return (silu(h @ _t(w, p + "gate").T) * (h @ _t(w, p + "up").T)) @ _t(w, p + "down").T


def moe(h: torch.Tensor, w, p: str, f: dict) -> torch.Tensor:
    r = f["router"]
    gr = r.get("groups") or {"count": 1, "keep": 1}
    z = h @ _t(w, p + "router").T
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, wt in route(z[t], r["top"], gr["count"], gr["keep"]):
            out[t] += wt * expert(h[t], w, p + f"e{e}.")
    return out


def softcap(z: torch.Tensor, cap: float) -> torch.Tensor:
    return cap * torch.tanh(z / cap)


def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens, layers_out: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] (float64) of one sequence; layers_out, if a list, receives the residual stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = _t(w, "embed")[torch.as_tensor(tokens, dtype=torch.long)]
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = tanh_norm(x, w, p + "norm1")
        if layer["type"] == "attention":
            x = x + attention_mixer(h, w, p + "mix.", m, eps)
        elif layer["type"] == "parallel":
            x = x + parallel_mixer(h, w, p + "mix.", m, eps)
        else:
            raise ValueError(layer["type"])
        if layer.get("mlp") is not None:
            x = x + moe(tanh_norm(x, w, p + "norm2"), w, p + "mlp.", layer["mlp"])
        if layers_out is not None:
            layers_out.append(x.clone())
    z = tanh_norm(x, w, "final.norm") @ _t(w, "head").T
    cap = cfg.get("logit_softcap")
    return softcap(z, cap) if cap else z
