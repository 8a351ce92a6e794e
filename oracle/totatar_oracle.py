"""Plain implementation of the Totatar design: float64, whole sequences, no cache, one function per mechanism.

It shares no code with the product path (`qspec_b200/totatar.py` and its kernels) and is the reference of the tests.
`cfg` is the dictionary of a config.json, `w` maps tensor names to torch tensors (any float type; read as float64).

    norm:       N(v; g) = v / sqrt(mean(v^2) + eps) * (1 + g)
    layer:      x <- x + N(mixer(N(x; norm1)); norm1b);   x <- x + N(ff(N(x; norm2)); norm2b)
    parallel:   left_scale * L(h) + right_scale * R(h)
      L         q, k, v = W h + b; q, k rotated (entry 2i with 2i + 1, frequencies divided by `factor`); softmax over the last `size`
                positions with exp(sink) in the denominator; W_o
      R         q, k, v = silu(W h); S <- decay S + k v^T; o = S^T q; W_o (unit_rms(o over all heads) * norm * sigmoid(W_g h))
    mamba2:     [z | x | B | C | dt] = W_in h; x, B, C = silu(conv + bias); dt = softplus(dt + dt_bias); per head
                S <- exp(-exp(A_log) dt) S + dt B x^T; y = S^T C + D x; W_o (unit_rms(y * silu(z), in equal parts) * norm)
    dense ff:   W_down (gelu_tanh(W_gate h) * (W_up h))
    moe ff:     z = W_router h + b; the largest z, softmax over those alone; sum of weight * expert(h), plus shared(h);
                expert(h) = W_down (silu(W_gate h) * (W_up h))
    end:        logits = embed N(x; final.norm)
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64


def _t(w: Dict[str, torch.Tensor], name: str) -> torch.Tensor:
    return w[name].to(F64)


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_centered(x: torch.Tensor, g: torch.Tensor, eps: float) -> torch.Tensor:
    """RMS norm whose weight is stored around zero."""
    return unit_rms(x, eps) * (1.0 + g)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.where(z > 30.0, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


# ---- parallel mixer, left half ------------------------------------------------------------------------------------------------

def frequencies(dims: int, base: float, factor: float = 1.0) -> List[float]:
    return [float(base) ** (-2.0 * i / dims) / factor for i in range(dims // 2)]


def rotate_interleaved(x: torch.Tensor, pos: torch.Tensor, freqs: List[float]) -> torch.Tensor:
    """x [T, heads, n]: entries 2i and 2i + 1 turn by pos * freqs[i]; the rest passes."""
    out = x.clone()
    for i, f in enumerate(freqs):
        a = pos.to(F64) * f
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def sink_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, size: Optional[int], sink: Optional[torch.Tensor]):
    """q [T, H, D], k [T, G, D], v [T, G, DV], sink [H] or None: softmax attention of position i over the j with 0 <= i - j < size
    (None: all j <= i), exp(sink_h) added to the denominator. Returns [T, H, DV]."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for t in range(T):
        lo = 0 if size is None else max(0, t - size + 1)
        for h in range(H):
            s = (k[lo:t + 1, h // rep] @ q[t, h]) * scale
            top = s.max() if sink is None else torch.maximum(s.max(), sink[h])
            e = torch.exp(s - top)
            total = e.sum() if sink is None else e.sum() + torch.exp(sink[h] - top)
            out[t, h] = (e / total) @ v[lo:t + 1, h // rep]
    return out


def left_mixer(h: torch.Tensor, w, p: str, m: dict) -> torch.Tensor:
    T = h.shape[0]
    H, G, D, DV = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (h @ _t(w, p + n).T + _t(w, p + n + ".b") for n in "qkv")
    q, k, v = q.view(T, H, D), k.view(T, G, D), v.view(T, G, DV)
    rot = m.get("rot") or {}
    if rot.get("dims"):
        fr = frequencies(rot["dims"], rot["base"], (rot.get("scaling") or {}).get("factor", 1.0))
        q, k = rotate_interleaved(q, torch.arange(T), fr), rotate_interleaved(k, torch.arange(T), fr)
    o = sink_attention(q, k, v, m["scale"], (m.get("mask") or {}).get("size"), _t(w, p + "sink"))
    return o.reshape(T, H * DV) @ _t(w, p + "o").T


# ---- parallel mixer, right half -----------------------------------------------------------------------------------------------

def scalar_decay(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, a: torch.Tensor, state: Optional[torch.Tensor] = None) -> torch.Tensor:
    """q, k [T, G, D], v [T, H, DV], a [T, H]: per head S <- a_t S + k_t v_t^T, o_t = S^T q_t; head h reads query / key head
    h // (H / G). Returns [T, H, DV]; `state` [H, D, DV], if given, is updated in place."""
    T, H, DV = v.shape
    rep = H // k.shape[1]
    S = torch.zeros(H, k.shape[2], DV, dtype=F64) if state is None else state
    o = torch.zeros(T, H, DV, dtype=F64)
    for t in range(T):
        for h in range(H):
            S[h] = a[t, h] * S[h] + torch.outer(k[t, h // rep], v[t, h])
            o[t, h] = S[h].T @ q[t, h // rep]
    return o


def right_mixer(h: torch.Tensor, w, p: str, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, D, DV = m["heads"], m["dim"], m["vdim"]
    q = silu(h @ _t(w, p + "q").T).view(T, H, D)
    k = silu(h @ _t(w, p + "k").T).view(T, H, D)
    v = silu(h @ _t(w, p + "v").T).view(T, H, DV)
    o = scalar_decay(q, k, v, torch.tensor(m["decay"], dtype=F64).expand(T, H)).reshape(T, H * DV)
    return (unit_rms(o, eps) * _t(w, p + "norm") * torch.sigmoid(h @ _t(w, p + "g").T)) @ _t(w, p + "o").T


def parallel_mixer(h: torch.Tensor, w, p: str, m: dict, eps: float) -> torch.Tensor:
    return m["left_scale"] * left_mixer(h, w, p + "left.", m["left"]) + m["right_scale"] * right_mixer(h, w, p + "right.", m["right"], eps)


# ---- mamba2 mixer -------------------------------------------------------------------------------------------------------------

def causal_conv(x: torch.Tensor, taps_w: torch.Tensor, bias: torch.Tensor) -> torch.Tensor:
    """x [T, C], taps_w [C, K]: y_t = bias + sum_j taps_w[:, j] * x_(t - K + 1 + j), zeros before the start."""
    T, K = x.shape[0], taps_w.shape[1]
    y = bias.expand(T, -1).clone()
    for t in range(T):
        for j in range(K):
            s = t - (K - 1) + j
            if s >= 0:
                y[t] += taps_w[:, j] * x[s]
    return y


def part_norm(y: torch.Tensor, parts: int, eps: float) -> torch.Tensor:
    """Every one of `parts` equal parts of a row by its own root mean square."""
    T, n = y.shape
    return unit_rms(y.view(T, parts, n // parts), eps).reshape(T, n)


def mamba2_mixer(h: torch.Tensor, w, p: str, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    z, xbc, dt = torch.split(h @ _t(w, p + "in").T, [inner, inner + 2 * G * N, H], dim=1)
    xbc = silu(causal_conv(xbc, _t(w, p + "conv"), _t(w, p + "conv.b")))
    x, B, C = torch.split(xbc, [inner, G * N, G * N], dim=1)
    x, B, C = x.reshape(T, H, P), B.reshape(T, G, N), C.reshape(T, G, N)
    dt = softplus(dt + _t(w, p + "dt_bias"))
    a = torch.exp(-torch.exp(_t(w, p + "A_log")) * dt)
    y = scalar_decay(C, B, dt[:, :, None] * x, a) + _t(w, p + "D")[:, None] * x
    y = y.reshape(T, inner) * silu(z)
    return (part_norm(y, m["norm_groups"], eps) * _t(w, p + "norm")) @ _t(w, p + "o").T


# ---- feed-forward -------------------------------------------------------------------------------------------------------------

def glu(h: torch.Tensor, w, p: str, act) -> torch.Tensor:
    return (act(h @ _t(w, p + "gate").T) * (h @ _t(w, p + "up").T)) @ _t(w, p + "down").T


def route(z: torch.Tensor, top: int):
    """One token's router logits [E] -> [(expert, weight)]: the largest ones, softmax over those alone."""
    chosen = sorted(range(len(z)), key=lambda e: (-float(z[e]), e))[:top]
    e = [math.exp(float(z[c]) - float(z[chosen[0]])) for c in chosen]
    return [(c, v / sum(e)) for c, v in zip(chosen, e)]


def moe(h: torch.Tensor, w, p: str, f: dict) -> torch.Tensor:
    z = h @ _t(w, p + "router").T + _t(w, p + "router.b")
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, wt in route(z[t], f["router"]["top"]):
            out[t] += wt * glu(h[t], w, p + f"e{e}.", silu)
    if f.get("shared"):
        out = out + glu(h, w, p + "shared.", silu)
    return out


def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens, layers_out: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] (float64) of one sequence; layers_out, if a list, receives the residual stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = _t(w, "embed")[torch.as_tensor(tokens, dtype=torch.long)]
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer.get("mlp")
        h = norm_centered(x, _t(w, p + "norm1"), eps)
        mixer = {"mamba2": mamba2_mixer, "parallel": parallel_mixer}[layer["type"]]
        x = x + norm_centered(mixer(h, w, p + "mix.", m, eps), _t(w, p + "norm1b"), eps)
        if f is not None:
            h = norm_centered(x, _t(w, p + "norm2"), eps)
            y = glu(h, w, p + "mlp.", gelu_tanh) if f["kind"] == "dense" else moe(h, w, p + "mlp.", f)
            x = x + norm_centered(y, _t(w, p + "norm2b"), eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return norm_centered(x, _t(w, "final.norm"), eps) @ _t(w, "embed").T
