"""Totatar on the GPU against the plain CPU restatement (oracle/totatar_oracle.py): every mechanism alone, then whole models through the
scheduler's step function -- whole prompts, token-by-token decoding, portions down to two tokens, mixed batches, reused slots, window
edges, far tokens, sinks, other sizes, long decoding and greedy generation."""
import json
import os

import pytest
import torch

from oracle import totatar_oracle as O

pytestmark = pytest.mark.gpu

F32, BF16, F64 = torch.float32, torch.bfloat16, torch.float64
FULL = 1 << 30


def _cuda():
    if not torch.cuda.is_available():
        pytest.skip("needs a CUDA device")
    from qspec_b200.build import build_seq_library
    build_seq_library()


def plan(segments, slots=4, max_step=4096):
    """segments: (slot, first position, count) or (slot, first position, count, phase) -> the step's BatchMeta."""
    from qspec_b200.state import SequenceTable
    t = SequenceTable(slots, "cuda", max_step)
    at = {t.open(("s", slot)): ("s", slot) for slot in range(slots)}
    for s in segments:
        t.pos[s[0]], t.phase[s[0]] = s[1], s[3] if len(s) > 3 else 0
    return t.plan([(at[s[0]], s[2]) for s in segments])


def rnd(g, *shape, dtype=F32, scale=1.0):
    """Random values that the element type represents exactly, as float64."""
    return (torch.randn(*shape, generator=g) * scale).to(dtype).to(F64)


def tol(dtype):
    return 2e-5 if dtype == F32 else 2.5e-2


def close(got, want, dtype, scale=None, bound=None):
    want = want.to(F64)
    s = float(want.abs().max()) if scale is None else scale
    err = float((got.detach().cpu().to(F64) - want).abs().max())
    assert err <= (bound or tol(dtype)) * max(s, 1e-6), f"max error {err:.3g} against scale {s:.3g}"


def dev(t, dtype=F32):
    return t.to(dtype).cuda().contiguous()


# ---------------------------------------------------------------------------------------------------------------------
# mechanisms alone
# ---------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("W", [40, 96, 257, 1100, 2052, 3001, 5000])
def test_residual_sum_between_two_norms(dtype, W):
    """One part; several weighted parts and an extra one; no sublayer at all; the sum without a norm after it."""
    _cuda()
    from qspec_b200 import ops
    g = torch.Generator().manual_seed(W)
    T, eps = 5, 1e-5
    x, y, y2 = rnd(g, T, W, scale=3.0), rnd(g, T, W, dtype=dtype), rnd(g, T, W, dtype=dtype)
    post, pre = rnd(g, W, scale=0.3), rnd(g, W, scale=0.3)
    y[1] *= 1e-3                                              # eps counts here
    y = y.to(dtype).to(F64)
    xo, out = torch.empty(T, W, dtype=F32, device="cuda"), torch.empty(T, W, dtype=dtype, device="cuda")
    ops.seq_sandwich_norm(dev(x), eps, y=dev(y, dtype), post_w=dev(post), pre_w=dev(pre), x_out=xo, out=out)
    r = x + O.norm_centered(y, post, eps)
    close(xo, r, F32)
    close(out, O.norm_centered(r, pre, eps), dtype)
    parts, wt = rnd(g, T, 3, W, dtype=dtype), rnd(g, T, 3)
    for extra in (None, y2):
        xi = dev(x)
        ops.seq_sandwich_norm(xi, eps, y=dev(parts, dtype), y_w=dev(wt), y2=dev(extra, dtype) if extra is not None else None, post_w=dev(post),
                              pre_w=dev(pre), x_out=xi, out=out)
        v = (parts * wt[:, :, None]).sum(1) + (extra if extra is not None else 0.0)
        r = x + O.norm_centered(v, post, eps)
        close(xi, r, F32)
        close(out, O.norm_centered(r, pre, eps), dtype)
    ops.seq_sandwich_norm(dev(x), eps, pre_w=dev(pre), out=out)
    close(out, O.norm_centered(x, pre, eps), dtype)
    ops.seq_sandwich_norm(dev(x), eps, y=dev(y, dtype), post_w=dev(post), x_out=xo, w_offset=0.0)
    close(xo, x + O.unit_rms(y, eps) * post, F32)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("N,parts", [(24, 1), (24, 3), (35, 5), (96, 2), (4096, 4), (1536, 1), (2310, 1), (9000, 3), (1030, 1)])
@pytest.mark.parametrize("mode", ["sigmoid_after", "silu_before"])
def test_gated_norm_in_parts(dtype, N, parts, mode):
    """Parts of very different size each have their own root mean square; the gate comes before or after; strided gate and output."""
    _cuda()
    from qspec_b200 import ops
    g = torch.Generator().manual_seed(N + parts)
    T, eps = 6, 1e-3
    src, w, wide = rnd(g, T, N), rnd(g, N), rnd(g, T, N + 12, dtype=dtype, scale=2.0)
    src.view(T, parts, -1).mul_(10.0 ** torch.arange(parts, dtype=F64)[None, :, None] * 0.01)
    src = src.to(F32).to(F64)
    gate = wide[:, 4:4 + N]
    buf = torch.full((T, N + 8), -1.0, dtype=dtype, device="cuda")
    ops.seq_part_norm(dev(src), dev(w), dev(wide, dtype)[:, 4:4 + N], mode, buf[:, 4:4 + N], eps, parts=parts, out_scale=1.25)
    u = src * O.silu(gate) if mode == "silu_before" else src
    want = 1.25 * O.part_norm(u, parts, eps) * w * (1.0 if mode == "silu_before" else torch.sigmoid(gate))
    close(buf[:, 4:4 + N], want, dtype)
    assert float((buf[:, :4] + 1.0).abs().max()) == 0.0 and float((buf[:, -4:] + 1.0).abs().max()) == 0.0


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("F", [1, 13, 64, 300])
def test_gated_linear_units(dtype, F):
    _cuda()
    from qspec_b200 import ops
    g = torch.Generator().manual_seed(F)
    gu = rnd(g, 9, 2 * F, dtype=dtype, scale=3.0)
    gu[0, 0], gu[1, 0] = 60.0, -60.0
    out = torch.empty(9, F, dtype=dtype, device="cuda")
    for name, act in (("silu", O.silu), ("gelu_tanh", O.gelu_tanh)):
        ops.seq_glu(dev(gu, dtype), out, name)
        close(out, act(gu[:, :F]) * gu[:, F:], dtype)
    if dtype == F32 and F == 300:                             # the tanh form, not the exact one
        exact = 0.5 * gu[:, :F] * (1.0 + torch.erf(gu[:, :F] / 2 ** 0.5)) * gu[:, F:]
        assert float((out.cpu().to(F64) - exact).abs().max()) > 1e-4


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("E,top", [(6, 2), (16, 3), (1, 1), (40, 5), (9, 9)])
def test_router_with_a_bias_and_a_softmax_over_the_chosen(dtype, E, top):
    """The bias is part of the logits: it changes the choice and the weights."""
    _cuda()
    from qspec_b200 import ops
    g = torch.Generator().manual_seed(E * 10 + top)
    T, W = 23, 36
    h, rw, b = rnd(g, T, W, dtype=dtype), rnd(g, E, W, scale=0.3), rnd(g, E, scale=2.0)
    idx, wt = torch.empty(T, top, dtype=torch.int32, device="cuda"), torch.empty(T, top, dtype=F32, device="cuda")
    ops.moe_route_chosen(dev(h, dtype), dev(rw), idx, wt, bias=dev(b))
    moved = False
    for t in range(T):
        want = O.route(rw @ h[t] + b, top)
        assert idx[t].tolist() == [e for e, _ in want]
        close(wt[t], torch.tensor([p for _, p in want], dtype=F64), F32)
        moved |= [e for e, _ in want] != [e for e, _ in O.route(rw @ h[t], top)]
    assert moved or E == 1


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("H,G,D,DV,dims,factor", [(4, 2, 16, 12, 12, 4.0), (3, 1, 10, 7, 4, 1.0), (2, 2, 7, 9, 0, 1.0), (6, 2, 64, 64, 64, 2.5),
                                                  (4, 1, 112, 40, 40, 8.0), (2, 1, 160, 96, 90, 1.0), (1, 1, 300, 301, 6, 3.0), (8, 1, 24, 20, 2, 2.0)])
def test_heads_without_a_norm_rotated_in_neighbouring_pairs(dtype, H, G, D, DV, dims, factor):
    """q, k and v at free columns of the row; the step crosses the ring's end and two sequences share it."""
    _cuda()
    from qspec_b200 import ops
    g = torch.Generator().manual_seed(H * 100 + D)
    cap = 13
    segs = [(2, 9, 9), (0, 0, 3), (1, 1040, 1)]
    T = sum(s[2] for s in segs)
    q_off, k_off, v_off, ld = 4, 4 + H * D + 3, 4 + H * D + 3 + G * D, 4 + H * D + 3 + G * (D + DV) + 5
    p = rnd(g, T, ld, dtype=dtype)
    pos = torch.tensor([p0 + i for _, p0, n in segs for i in range(n)])
    fr = O.frequencies(dims, 60.0, factor) if dims else []
    q, k = p[:, q_off:q_off + H * D].reshape(T, H, D), p[:, k_off:k_off + G * D].reshape(T, G, D)
    q, k, v = O.rotate_interleaved(q, pos, fr), O.rotate_interleaved(k, pos, fr), p[:, v_off:v_off + G * DV].reshape(T, G, DV)
    ck = torch.full((4, cap, G, D), 9.0, dtype=dtype, device="cuda")
    cv = torch.full((4, cap, G, DV), 9.0, dtype=dtype, device="cuda")
    qo = torch.empty(T, H, D, dtype=F32, device="cuda")
    ops.seq_head_prep(dev(p, dtype), q_off, k_off, v_off, qo, ck, cv, plan(segs).table, H, 1e-5, norm=False, pairing="interleaved",
                      inv_freq=dev(torch.tensor(fr)) if dims else None, rot_dims=dims)
    angle = 2e-4 if dtype == F32 else None                    # position 1040 in float32 radians
    close(qo, q, F32, bound=angle)
    at, touched = 0, set()
    for slot, p0, n in segs:
        for i in range(n):
            close(ck[slot, (p0 + i) % cap], k[at], dtype, bound=angle)
            close(cv[slot, (p0 + i) % cap], v[at], dtype)
            touched.add((slot, (p0 + i) % cap))
            at += 1
    for slot in range(4):
        for r in range(cap):
            if (slot, r) not in touched:
                assert float((ck[slot, r] - 9.0).abs().max()) == 0.0 and float((cv[slot, r] - 9.0).abs().max()) == 0.0


@pytest.mark.parametrize("vec", [True, False])
def test_the_older_head_forms_keep_their_meaning(vec):
    """Halves pairing with a norm before the rotation, as the default arguments give it."""
    _cuda()
    from qspec_b200 import ops
    from oracle import legavik_oracle as L
    g = torch.Generator().manual_seed(2)
    H, G, D, DV, dims, T = 2, 1, (16 if vec else 10), (8 if vec else 7), 6, 5
    p = rnd(g, T, (H + G) * D + G * DV)
    fr = L.yarn_frequencies(dims, 40.0, None)
    q = L.rotate_halves(L.unit_rms(p[:, :H * D].reshape(T, H, D), 1e-5), torch.arange(T), fr, 1.0)
    ck, cv = torch.zeros(1, 8, G, D, device="cuda"), torch.zeros(1, 8, G, DV, device="cuda")
    qo = torch.empty(T, H, D, dtype=F32, device="cuda")
    ops.seq_head_prep(dev(p), 0, H * D, (H + G) * D, qo, ck, cv, plan([(0, 0, T)], slots=1).table, H, 1e-5, inv_freq=dev(torch.tensor(fr)), rot_dims=dims)
    close(qo, q, F32)


# ---- window attention with a sink -----------------------------------------------------------------------------------------------
def _ring(rows, slot, slots, cap, dtype):
    """Cache [slots, cap, G, n] whose slot holds the rows of positions 0, 1, ... (later ones over earlier ones), all else 1e4."""
    c = torch.full((slots, cap) + tuple(rows.shape[1:]), 1e4, dtype=dtype, device="cuda")
    for j in range(rows.shape[0]):
        c[slot, j % cap] = rows[j].to(dtype).cuda()
    return c


def _attend(form, q, ck, cv, out, meta, window, scale, **kw):
    from qspec_b200 import ops
    if form == "plain":
        ops.seq_window_attention(q, None, ck, cv, out, meta.table, window, scale, **kw)
    elif form == "tile":
        (_, slot, first, _), = meta.segments
        ops.seq_prompt_attention_mma(q, ck, None, cv, out, slot, first, window, scale, **kw)
    else:
        ops.seq_window_attention_mma(q, ck, None, cv, out, meta.table, window, scale, form == "rows", **kw)


FORMS = [("plain", F32, (4, 2, 12, 10)), ("plain", F32, (3, 1, 80, 56)), ("plain", BF16, (5, 1, 112, 33)), ("heads", BF16, (8, 1, 64, 64)),
         ("heads", BF16, (4, 2, 128, 64)), ("rows", BF16, (4, 2, 64, 128)), ("tile", BF16, (2, 1, 64, 64)), ("tile", BF16, (2, 1, 128, 128))]


@pytest.mark.parametrize("form,dtype,sizes", FORMS)
@pytest.mark.parametrize("window", [1, 9, 70, FULL])
def test_window_attention_with_a_sink(form, dtype, sizes, window):
    """Portions that start anywhere in a ring that has wrapped, sinks below, among and far above the scores, a strided output, a factor."""
    _cuda()
    H, G, D, DV = sizes
    g = torch.Generator().manual_seed(window % 1000 + D)
    n, scale = 150, 0.4 * D ** -0.5
    q, k, v = rnd(g, n, H, D), rnd(g, n, G, D, dtype=dtype), rnd(g, n, G, DV, dtype=dtype)
    sink = torch.linspace(-3.0, 6.0, H, dtype=F64)
    want = 1.25 * O.sink_attention(q, k, v, scale, None if window == FULL else window, sink)
    without = 1.25 * O.sink_attention(q, k, v, scale, None if window == FULL else window, None)
    top = float(want.abs().max())
    assert float((want - without)[:, -1].abs().max()) > 0.2 * float(without.abs().max())       # the sink shows
    for first, count in ((0, 40), (0, 1), (33, 64), (100, 50), (149, 1)):
        if form == "tile" and count == 1:
            continue
        end = first + count
        cap = n if window == FULL else window - 1 + count
        ck, cv = _ring(k[:end], 1, 3, cap, dtype), _ring(v[:end], 1, 3, cap, dtype)
        wide = torch.full((count, H * DV + 8), -1.0, dtype=dtype, device="cuda")
        out = wide.as_strided((count, H, DV), (H * DV + 8, DV, 1), 4) if form == "plain" else wide.as_strided((count, H, DV), (H * DV + 8, DV, 1), 8)
        _attend(form, dev(q[first:end]), ck, cv, out, plan([(1, first, count)]), window, scale, sink=dev(sink), out_scale=1.25)
        close(out, want[first:end], dtype, scale=top)


@pytest.mark.parametrize("form,dtype,sizes", [FORMS[1], FORMS[2], ("heads", BF16, (2, 1, 64, 64)), ("rows", BF16, (2, 1, 64, 64)), FORMS[6]])
@pytest.mark.parametrize("inside", [True, False])
def test_a_key_that_stands_out_at_the_edge_of_the_window(form, dtype, sizes, inside):
    """One key matches the last query far better than the others and its value stands out: in the window's last place the output carries
    it, one place further back it does not. In portions and alone."""
    _cuda()
    H, G, D, DV = sizes
    g = torch.Generator().manual_seed(17)
    n, window = 300, 100
    q, k, v = rnd(g, n, H, D, scale=0.3), rnd(g, n, G, D, dtype=dtype, scale=0.3), rnd(g, n, G, DV, dtype=dtype, scale=0.1)
    j = n - window if inside else n - 1 - window
    k[j, 0] = (q[n - 1, 1] * 8.0).to(dtype).to(F64)
    v[j, 0] = 5.0
    sink = torch.zeros(H, dtype=F64)
    want = O.sink_attention(q, k, v, 1.0, window, sink)
    assert (float(want[n - 1, 1].mean()) > 2.0) == inside
    cap = window - 1 + 30
    ck, cv = _ring(k, 0, 2, cap, dtype), _ring(v, 0, 2, cap, dtype)
    for count in (30, 1):
        if form == "tile" and count == 1:
            continue
        out = torch.empty(count, H, DV, dtype=dtype, device="cuda")
        _attend(form, dev(q[n - count:]), ck, cv, out, plan([(0, n - count, count)]), window, 1.0, sink=dev(sink))
        close(out, want[n - count:], dtype, scale=float(want[n - count:].abs().max()))
        assert (float(out[-1, 1].float().mean()) > 2.0) == inside


# ---- short convolution in runs of tokens ----------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("C,taps", [(8, 4), (12, 1), (8, 3), (20, 2), (1028, 4)])
@pytest.mark.parametrize("n", [900, 30])
def test_convolution_over_runs_of_tokens(dtype, C, taps, n):
    """Enough tokens for several per thread, segments that begin and end inside such a run or are shorter than the filter, strided rows,
    both tail buffers."""
    _cuda()
    from qspec_b200 import ops
    if C > 1000 and n > 100:
        n = 400
    g = torch.Generator().manual_seed(C + taps)
    lens = [(0, 0, 2 * n + 3, 0), (1, 5, n - 5, 1), (2, 2, 1, 0), (3, 1, 3, 1)] if n > 100 else [(0, 0, n, 0), (1, 2, 1, 1), (2, 40, 5, 0), (3, 0, 2, 1)]
    w, b = rnd(g, C, taps), rnd(g, C)
    hist = {s: rnd(g, p0, C) for s, p0, _, _ in lens}
    x = {s: rnd(g, m, C, dtype=dtype) for s, _, m, _ in lens}
    tail = torch.full((2, 4, taps - 1, C), 1e4, dtype=F32, device="cuda")
    for s, p0, _, ph in lens:
        for r in range(taps - 1):
            j = p0 - (taps - 1) + r
            if j >= 0:
                tail[ph, s, r] = hist[s][j].to(F32).cuda()
    meta = plan(lens)
    wide = torch.zeros(meta.ntok, C + 12, dtype=dtype, device="cuda")
    wide[:, 4:4 + C] = dev(torch.cat([x[s] for s, _, _, _ in lens]), dtype)
    out = torch.empty(meta.ntok, C, dtype=dtype, device="cuda")
    ops.seq_conv_act(wide[:, 4:4 + C], dev(w), dev(b), tail, out, meta.table, act="silu")
    at = 0
    for s, p0, m, ph in lens:
        full = torch.cat([hist[s], x[s]])
        lo = max(0, p0 - taps)
        want = O.silu(O.causal_conv(full[lo:], w, b))[p0 - lo:] if p0 else O.silu(O.causal_conv(full, w, b))
        close(out[at:at + m], want, dtype, scale=4.0)
        for r in range(taps - 1):
            j = p0 + m - (taps - 1) + r
            close(tail[1 - ph, s, r], full[j] if j >= 0 else torch.zeros(C, dtype=F64), F32)
        at += m


# ---- matrix states with one decay per head and token ----------------------------------------------------------------------------
def _fixed(decay):
    import math
    return dict(decay=dev(torch.tensor(decay)), log_decay=dev(torch.tensor([math.log(v) if v > 0 else -1e30 for v in decay])))


@pytest.mark.parametrize("dtype,chunks", [(F32, False), (BF16, False), (BF16, True)])
@pytest.mark.parametrize("H,D,DV", [(4, 16, 24), (3, 7, 5), (1, 64, 64), (2, 128, 96), (2, 72, 136), (1, 200, 40), (2, 256, 8), (5, 33, 130),
                                    (2, 300, 12), (1, 700, 9)])
def test_linear_attention_with_fixed_decays(dtype, H, D, DV, chunks):
    """Portions of many lengths with the state carried over, in two sequences at a time, one of them fresh in a slot full of NaN; decays
    of one, zero and between."""
    _cuda()
    from qspec_b200 import ops
    g = torch.Generator().manual_seed(D * DV)
    decay = [0.999, 0.5, 1.0, 0.0, 0.93][:H]
    n, m = 230, 60
    ld = 3 + H * (2 * D + DV)
    ld += -ld % 8
    q_off, k_off, v_off = 0, H * D, 2 * H * D
    A, B = rnd(g, n, ld, dtype=dtype, scale=0.8), rnd(g, m, ld, dtype=dtype, scale=0.8)

    def want(p):
        sec = lambda o, w: O.silu(p[:, o:o + H * w]).view(-1, H, w)
        return O.scalar_decay(sec(q_off, D), sec(k_off, D), sec(v_off, DV), torch.tensor(decay, dtype=F64).expand(p.shape[0], H)).reshape(-1, H * DV)

    wa, wb = want(A), want(B)
    state = torch.full((4, H, D, DV), float("nan"), dtype=F32, device="cuda")
    scratch = torch.empty(max(ops.seq_scalar_decay_scratch_bytes(16, H, D, DV), 16), dtype=torch.uint8, device="cuda") if chunks else None
    at = {"a": 0, "b": 0}
    for na, nb in ((40, 0), (2, 33), (65, 1), (1, 3), (7, 0), (64, 23), (51, 0)):
        segs = ([(1, at["a"], na)] if na else []) + ([(3, at["b"], nb)] if nb else [])
        meta = plan(segs)
        p = dev(torch.cat([A[at["a"]:at["a"] + na], B[at["b"]:at["b"] + nb]]), dtype)
        y = torch.empty(na + nb, H * DV, dtype=F32, device="cuda")
        ops.seq_scalar_decay(p, q_off, k_off, v_off, H, state, y, meta, scratch=scratch, **_fixed(decay))
        bound = 2e-5 if dtype == F32 else 1.2e-2
        close(y[:na], wa[at["a"]:at["a"] + na], dtype, scale=float(wa.abs().max()), bound=bound)
        if nb:
            close(y[na:], wb[at["b"]:at["b"] + nb], dtype, scale=float(wb.abs().max()), bound=bound)
        at["a"] += na
        at["b"] += nb
    assert at == {"a": n, "b": m} and bool(torch.isnan(state[0]).all()) and bool(torch.isnan(state[2]).all())


def _ssm(g, T, H, G, N, P, taps, dtype, dt_scale=1.0):
    """A random Mamba-2 recurrence: rows [z | x | B | C | dt] on boundaries of eight, its weights, and the columns."""
    up = lambda v: v + -v % 8
    x = up(H * P)
    cols = {"x": x, "B": 2 * x, "C": 2 * x + up(G * N), "dt": 2 * x + 2 * up(G * N)}
    p = rnd(g, T, cols["dt"] + up(H), dtype=dtype)
    Cn = cols["dt"] - cols["x"]
    wt = {"conv": rnd(g, Cn, taps, scale=0.6), "b": rnd(g, Cn, scale=0.3), "dt_bias": rnd(g, H) * dt_scale, "A_log": rnd(g, H) * 0.7, "D": rnd(g, H)}
    return cols, p, wt


def _ssm_want(cols, p, wt, H, G, N, P, act_dtype):
    T = p.shape[0]
    act = O.silu(O.causal_conv(p[:, cols["x"]:cols["dt"]], wt["conv"], wt["b"])).to(act_dtype).to(F64)
    o = cols["x"]
    x, B, C = (act[:, cols[n] - o:cols[n] - o + w].reshape(T, -1, d) for n, w, d in (("x", H * P, P), ("B", G * N, N), ("C", G * N, N)))
    dt = O.softplus(p[:, cols["dt"]:cols["dt"] + H] + wt["dt_bias"])
    y = O.scalar_decay(C, B, dt[:, :, None] * x, torch.exp(-torch.exp(wt["A_log"]) * dt)) + wt["D"][:, None] * x
    return y.reshape(T, H * P)


@pytest.mark.parametrize("dtype,chunks", [(F32, False), (BF16, False), (BF16, True)])
@pytest.mark.parametrize("H,G,N,P,taps,dt_scale", [(4, 2, 16, 24, 4, 1.0), (3, 1, 7, 5, 2, 1.0), (2, 2, 64, 64, 1, 1.0), (4, 1, 128, 32, 3, 30.0),
                                                   (2, 1, 40, 8, 6, 1.0), (6, 3, 24, 72, 4, 30.0), (1, 1, 256, 16, 4, 1.0), (2, 1, 272, 6, 3, 1.0)])
def test_mamba2_recurrence_with_its_convolution(dtype, H, G, N, P, taps, dt_scale, chunks):
    """Portions of many lengths, down to single tokens and shorter than the filter, of two sequences; step sizes up to hundreds (decays
    far below the smallest float32); used tails and states."""
    _cuda()
    from qspec_b200 import ops
    g = torch.Generator().manual_seed(N * P + taps)
    cols, A, wt = _ssm(g, 200, H, G, N, P, taps, dtype, dt_scale)
    B = rnd(g, 50, A.shape[1], dtype=dtype)
    wa, wb = (_ssm_want(cols, p, wt, H, G, N, P, dtype) for p in (A, B))
    Cn = cols["dt"] - cols["x"]
    state = torch.full((4, H, N, P), float("nan"), dtype=F32, device="cuda")
    tail = torch.full((2, 4, taps - 1, Cn), 1e4, dtype=F32, device="cuda")
    scratch = torch.empty(max(ops.seq_scalar_decay_scratch_bytes(16, H, N, P), 16), dtype=torch.uint8, device="cuda") if chunks else None
    w = {k: dev(v) for k, v in wt.items()}
    at, ph = {"a": 0, "b": 0}, {"a": 0, "b": 1}
    for na, nb in ((3, 0), (40, 1), (1, 34), (66, 1), (2, 14), (1, 0), (87, 0)):
        segs = ([(1, at["a"], na, ph["a"])] if na else []) + ([(2, at["b"], nb, ph["b"])] if nb else [])
        meta = plan(segs)
        p = dev(torch.cat([A[at["a"]:at["a"] + na], B[at["b"]:at["b"] + nb]]), dtype)
        y = torch.empty(na + nb, H * P, dtype=F32, device="cuda")
        ops.seq_scalar_decay(p, cols["C"], cols["B"], cols["x"], G, state, y, meta, dt=p[:, cols["dt"]:cols["dt"] + H], dt_bias=w["dt_bias"],
                             A_log=w["A_log"], D_skip=w["D"], conv=(w["conv"], w["b"], cols["x"], tail),
                             conv_out=torch.empty(na + nb, Cn, dtype=dtype, device="cuda"), scratch=scratch)
        bound = 2e-5 if dtype == F32 else 6e-3
        close(y[:na], wa[at["a"]:at["a"] + na], dtype, scale=float(wa.abs().max()), bound=bound)
        if nb:
            close(y[na:], wb[at["b"]:at["b"] + nb], dtype, scale=float(wb.abs().max()), bound=bound)
        for s, k in (("a", na), ("b", nb)):
            at[s] += k
            ph[s] ^= 1 if k else 0
    assert at == {"a": 200, "b": 50}


@pytest.mark.parametrize("form", ["chunks", "tokens", "float32"])
def test_a_token_far_back_in_the_state(form):
    """Only token 3 of 700 writes along the axis that the late queries read; decays close to one. The read-outs agree to the accuracy of
    float32 states -- rounding the state to bfloat16 anywhere would show."""
    _cuda()
    from qspec_b200 import ops
    dtype = F32 if form == "float32" else BF16
    g = torch.Generator().manual_seed(5)
    n, H, D, DV = 700, 2, 64, 64
    decay = [0.9995, 1.0]
    p = rnd(g, n, H * (2 * D + DV), dtype=dtype)
    q, k, v = p[:, :H * D].view(n, H, D), p[:, H * D:2 * H * D].view(n, H, D), p[:, 2 * H * D:].view(n, H, DV)
    k[:, :, 11] = 0.0
    q[650:] = 0.0
    k[3, :, 11], q[650:, :, 11] = 1.0, 1.0
    want = O.scalar_decay(q, k, v, torch.tensor(decay, dtype=F64).expand(n, H)).reshape(n, H * DV)
    assert float((want[699, DV:] - v[3, 1]).abs().max()) < 1e-9
    state = torch.zeros(1, H, D, DV, dtype=F32, device="cuda")
    scratch = torch.empty(ops.seq_scalar_decay_scratch_bytes(16, H, D, DV), dtype=torch.uint8, device="cuda") if form == "chunks" else None
    for cuts in ([700], [300, 64, 1, 2, 333]):
        at = 0
        state.fill_(7.0)
        for c in cuts:
            y = torch.empty(c, H * DV, dtype=F32, device="cuda")
            ops.seq_scalar_decay(dev(p[at:at + c], dtype), 0, H * D, 2 * H * D, H, state, y, plan([(0, at, c)], slots=1), silu=False,
                                 scratch=scratch, **_fixed(decay))
            close(y, want[at:at + c], F32, scale=float(want[at:at + c].abs().max()), bound=1e-4)
            if at + c == n:                                    # the rows that read token 3 alone, at its own scale
                close(y[-50 if c >= 50 else -c:], want[-50 if c >= 50 else -c:], F32, scale=1.0, bound=2e-3)
            at += c


# ---------------------------------------------------------------------------------------------------------------------
# whole models through the scheduler
# ---------------------------------------------------------------------------------------------------------------------
def parallel(left=(4, 2, 16, 12), window=20, dims=8, base=500.0, factor=4.0, right=(4, 12, 10), decay=None, scales=(0.8, 1.25), scale=0.25):
    lh, lg, ld, lv = left
    rh, rd, rv = right
    decay = decay or [0.999, 0.5, 0.93, 0.98, 1.0, 0.8][:rh]
    lm = {"heads": lh, "kv_heads": lg, "dim": ld, "vdim": lv, "scale": scale}
    if window:
        lm["mask"] = {"size": window}
    if dims:
        lm["rot"] = {"base": base, "dims": dims, "scaling": {"factor": factor}}
    return {"type": "parallel", "mixer": {"left": lm, "right": {"heads": rh, "dim": rd, "vdim": rv, "decay": decay},
                                          "left_scale": scales[0], "right_scale": scales[1]}}


def mamba2(heads=4, groups=2, state=16, vdim=12, conv=4, norm_groups=2):
    return {"type": "mamba2", "mixer": {"heads": heads, "groups": groups, "state": state, "vdim": vdim, "conv": conv, "norm_groups": norm_groups}}


def moe(ff=24, experts=8, top=3, shared=20):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}, "shared": {"ff": shared} if shared else None}


def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def config(layers, width=64, vocab=97, eps=1e-5):
    return {"architecture": "Totatar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


CONFIGS = {
    # every mixer with every feed-forward, windows shorter and longer than the portions
    "mixed": config([dict(parallel(), mlp=dense()), dict(mamba2(), mlp=moe()), dict(mamba2(heads=6, groups=3, state=24, vdim=8, norm_groups=3), mlp=None),
                     dict(parallel(left=(6, 1, 24, 8), window=33, dims=24, right=(2, 16, 24)), mlp=moe(ff=16, experts=6, top=2)),
                     dict(mamba2(heads=2, groups=1, state=40, vdim=16, conv=2, norm_groups=1), mlp=dense(24))]),
    # nothing divisible by anything: single heads, a window of one token, no rotation, one-tap and long filters, as many norm groups as
    # entries allow, one expert, as many chosen as there are, no shared expert, a model that opens and closes with the scan
    "odd": config([dict(mamba2(heads=3, groups=1, state=7, vdim=5, conv=1, norm_groups=5), mlp=moe(ff=13, experts=5, top=1, shared=0)),
                   dict(parallel(left=(3, 3, 10, 7), window=1, dims=0, right=(1, 33, 7), scales=(1.0, 1.0)), mlp=None),
                   dict(parallel(left=(5, 1, 6, 9), window=9, dims=2, base=37.0, factor=1.0, right=(3, 5, 17)), mlp=moe(ff=9, experts=3, top=3, shared=11)),
                   dict(mamba2(heads=5, groups=5, state=33, vdim=3, conv=6, norm_groups=3), mlp=dense(17))], width=50, vocab=33, eps=1e-6),
    # sizes of the tensor-core forms: attention heads of 64 and 128, chunks of the recurrences with several slices of values
    "wide": config([dict(parallel(left=(4, 2, 64, 64), window=48, dims=32, right=(2, 64, 128), scale=0.12), mlp=moe(ff=32, shared=32)),
                    dict(mamba2(heads=4, groups=1, state=128, vdim=64, norm_groups=4), mlp=dense(64)),
                    dict(parallel(left=(4, 1, 128, 128), window=70, dims=128, right=(1, 136, 72), scale=0.08), mlp=None),
                    dict(mamba2(heads=2, groups=2, state=64, vdim=96, norm_groups=1), mlp=moe(ff=32, experts=4, top=2, shared=0))], width=96),
    # attention over the whole sequence
    "full": config([dict(parallel(window=None), mlp=moe()), dict(mamba2(), mlp=None)]),
}


def build(name, dtype, seed=0, n_slots=3, max_step_tokens=64, max_seq_tokens=None):
    _cuda()
    from qspec_b200.scheduler import Scheduler
    from qspec_b200.totatar import TotatarConfig, TotatarModel, random_weights
    d = CONFIGS[name]
    cfg = TotatarConfig.from_dict(d)
    w = random_weights(cfg, seed)
    model = TotatarModel(cfg, w, dtype=dtype, device="cuda", n_slots=n_slots, max_step_tokens=max_step_tokens, max_seq_tokens=max_seq_tokens)
    model.prompt_tiles_min_ctas = 2                        # short test prompts take the tile form too
    return d, w, model, Scheduler(model)


def tokens(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def close_logits(got, ref, dtype, same_format=False):
    """Per position: root mean square over the vocabulary of the difference (mean taken off), relative to the spread of the
    logits. float32 against the plain implementation: rounding level. bfloat16 against the plain implementation: what an 8-bit
    mantissa leaves, with a few positions further off where two experts' logits are nearly equal. same_format: bfloat16 against
    bfloat16 logits of the same model fed another way."""
    ref = ref.to(F64)
    d = got.detach().cpu().to(F64) - ref
    d = d - d.mean(-1, keepdim=True)
    spread = float((ref - ref.mean(-1, keepdim=True)).pow(2).mean().sqrt())
    rows = d.pow(2).mean(-1).sqrt() / spread
    if dtype == F32:
        assert float(rows.median()) <= 1e-5, f"median position: {float(rows.median()):.3g} of the logits' spread"
        assert float(rows.max()) <= 3e-4, f"worst position: {float(rows.max()):.3g} of the logits' spread"
        return
    bound = 1.5e-2 if same_format else 3e-2
    assert float(rows.median()) <= bound, f"median position: {float(rows.median()):.3g} of the logits' spread"
    over = float((rows > 0.1).float().mean())
    assert over <= 0.1, f"{over:.1%} of the positions are off by more than 10% of the logits' spread"


_PLAIN = {}


def plain(name, toks, seed=0, layers=None):
    """The plain implementation's logits, computed once per model and sequence."""
    key = (name, seed, tuple(toks))
    if key not in _PLAIN:
        from qspec_b200.totatar import TotatarConfig, random_weights
        lay = []
        _PLAIN[key] = (O.forward(CONFIGS[name], random_weights(TotatarConfig.from_dict(CONFIGS[name]), seed), toks, lay), lay)
    if layers is not None:
        layers.extend(_PLAIN[key][1])
    return _PLAIN[key][0]


def reference_logits(name, toks, dtype):
    """float32: the plain implementation. bfloat16: the same weights in a second model that takes the prompt whole, after that
    has been held against the plain implementation."""
    ref = plain(name, toks)
    if dtype == F32:
        return ref
    _, _, _, s = build(name, dtype, max_step_tokens=256)
    whole = s.feed([("whole", toks, list(range(len(toks))))]).float().cpu()
    close_logits(whole, ref, dtype)
    return whole


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_matches_the_plain_implementation(name, dtype):
    cfg, w, model, s = build(name, dtype, max_step_tokens=128)
    toks = tokens(110, cfg["vocab"], 1)
    lay = []
    ref = plain(name, toks, layers=lay)
    close_logits(s.feed([("a", toks, list(range(len(toks))))]), ref, dtype)
    if dtype == F32:                                       # residual stream after every layer
        meta = s.table.plan([("b", len(toks))])
        tr = []
        model.forward_batch(torch.tensor(toks, dtype=torch.int32, device="cuda"), meta, trace=tr)
        assert len(tr) == len(lay) == len(cfg["layers"])
        for a, b in zip(tr, lay):
            close(a, b, F32)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_decoding_and_portions_equal_the_whole_prompt(name, dtype):
    """Token by token from the first token on; a prompt then 40 single tokens; portions of 2, 3, 1, 7, ... tokens, some long enough for
    the chunk form; a step longer than the model's step size (cut inside the step function)."""
    cfg, w, model, s = build(name, dtype, max_step_tokens=48)
    toks = tokens(110, cfg["vocab"], 1)
    ref = reference_logits(name, toks, dtype)
    schedules = {"single": [1] * len(toks), "prompt+decode": [48, 20, 2] + [1] * 40, "twos": [2] * 55,
                 "portions": [2, 3, 1, 7, 2, 34, 2, 5, 2, 40, 9, 3], "one step": [len(toks)]}
    for label, cuts in schedules.items():
        assert sum(cuts) == len(toks)
        at, rows = 0, []
        for n in cuts:
            rows.append(s.feed([(label, toks[at:at + n], list(range(n)))]))
            at += n
        s.release(label)
        close_logits(torch.cat(rows), ref, dtype, same_format=True)


@pytest.mark.parametrize("name", ["mixed", "wide", "odd"])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_mixed_batches_equal_each_request_alone_and_slots_are_reused(name, dtype):
    """Three requests of unequal length advance together -- a prompt portion next to single tokens next to a request that
    starts late in a slot another request has just given back -- and each must see what it sees alone."""
    cfg, w, model, s = build(name, dtype, n_slots=2, max_step_tokens=80)
    seqs = {"a": tokens(90, cfg["vocab"], 11), "b": tokens(23, cfg["vocab"], 12), "c": tokens(71, cfg["vocab"], 13)}
    alone = {}
    for rid, toks in seqs.items():
        alone[rid] = s.feed([(rid, toks, list(range(len(toks))))]).float().cpu()
        s.release(rid)
        if dtype == F32:
            close_logits(alone[rid], plain(name, toks), dtype)
    sched = [{"a": 7, "b": 20}, {"a": 1, "b": 1}, {"a": 40, "b": 2}, {"a": 1}, {"a": 1, "c": 9}, {"a": 2, "c": 1}, {"a": 38, "c": 35}, {"c": 26}]
    at = {k: 0 for k in seqs}
    got = {k: [] for k in seqs}
    for stepn, st in enumerate(sched):
        entries = [(rid, seqs[rid][at[rid]:at[rid] + n], list(range(n))) for rid, n in st.items()]
        out = s.feed(entries)
        o = 0
        for rid, n in st.items():
            got[rid].append(out[o:o + n].float().cpu())
            o += n
            at[rid] += n
        if stepn == 2:
            assert at["b"] == len(seqs["b"])
            s.release("b")                                  # request c takes this slot in the step after next
    for rid in seqs:
        assert at[rid] == len(seqs[rid])
        close_logits(torch.cat(got[rid]), alone[rid], dtype, same_format=True)


def test_stale_caches_states_and_tails_do_not_matter():
    """Everything a slot holds is overwritten with other numbers between two requests."""
    cfg, w, model, s = build("mixed", F32, n_slots=1, max_step_tokens=32)
    toks = tokens(50, cfg["vocab"], 3)
    ref = plain("mixed", toks)
    for value in (1e4, -3.0):
        for d in (model.cache_k, model.cache_v, model.rec_state, model.tail):
            for t in d.values():
                t.fill_(value)
        rows = [s.feed([("r", toks[:30], list(range(30)))])] + [s.feed([("r", [t], [0])]) for t in toks[30:]]
        s.release("r")
        close_logits(torch.cat(rows), ref, F32)


def test_batch_composition_changes_nothing_in_float32():
    """The same token of the same request, once alone in its step and once between two other requests: every kernel assigns work
    by position and size alone, so the logits agree to the last rounding of the vendor's matrix products."""
    cfg, w, model, s = build("odd", F32, n_slots=3, max_step_tokens=64)
    a, b, c = tokens(20, cfg["vocab"], 21), tokens(9, cfg["vocab"], 22), tokens(14, cfg["vocab"], 23)
    assert s.feed([("a", a[:19], []), ("b", b[:8], []), ("c", c[:13], [])]).shape[0] == 0
    mixed = s.feed([("b", b[8:], [0]), ("a", a[19:], [0]), ("c", c[13:], [0])])[1].float().cpu()
    for rid in "abc":
        s.release(rid)
    s.feed([("a", a[:19], [])])
    alone = s.feed([("a", a[19:], [0])])[0].float().cpu()
    assert float((mixed - alone).abs().max()) <= 2e-5 * float(alone.abs().max())


@pytest.mark.parametrize("half", ["left", "right"])
def test_each_half_of_a_parallel_layer_alone(half):
    """With one half's scale at zero the other one is all there is: the silent half's weights must not matter, its state and
    biases included."""
    from qspec_b200.scheduler import Scheduler
    from qspec_b200.totatar import TotatarConfig, TotatarModel, random_weights
    _cuda()
    scales = (1.5, 0.0) if half == "left" else (0.0, 1.5)
    d = config([dict(parallel(scales=scales), mlp=None), dict(parallel(scales=scales), mlp=moe())])
    w = random_weights(TotatarConfig.from_dict(d), 4)
    toks = tokens(40, 97, 4)
    ref = O.forward(d, w, toks)
    other = "right" if half == "left" else "left"
    w2 = {k: (v.flip(0) * 2.0 if f".{other}." in k else v) for k, v in w.items()}
    for ww in (w, w2):
        m = TotatarModel(TotatarConfig.from_dict(d), ww, dtype=F32, device="cuda", n_slots=1, max_step_tokens=20)
        close_logits(Scheduler(m).feed([("a", toks, list(range(40)))]), ref, F32)


def test_the_ring_is_short_and_the_sequence_unbounded():
    """Window layers alone do not bound the sequence: the rings hold the window and a step; far beyond them, prompts and decoding still
    equal the plain implementation."""
    cfg, w, m, s = build("mixed", F32, n_slots=2, max_step_tokens=10)
    assert m.max_seq_len is None and m.cache_k[0].shape[1] == 20 - 1 + 10 and m.cache_k[3].shape[1] == 33 - 1 + 10
    toks = tokens(160, 97, 7)
    ref = plain("mixed", toks)
    for label, cuts in (("whole", [160]), ("decode", [70] + [1] * 90), ("portions", [10, 2, 3, 10, 7] * 5)):
        at, rows = 0, []
        for n in cuts:
            rows.append(s.feed([(label, toks[at:at + n], list(range(n)))]))
            at += n
        close_logits(torch.cat(rows), ref, F32)
        s.release(label)


def test_attention_over_the_whole_sequence_bounds_it():
    cfg, w, model, s = build("full", BF16, max_seq_tokens=40)
    s.feed([("a", tokens(40, cfg["vocab"], 5), [39])])
    with pytest.raises(RuntimeError):
        s.feed([("a", [1], [0])])


def test_long_decoding():
    """A short prompt, then 230 single tokens: windows pass over decoded tokens several times, the recurrences' states go on, against the
    plain implementation."""
    cfg, w, model, s = build("mixed", F32, max_step_tokens=8)
    toks = tokens(250, cfg["vocab"], 6)
    ref = plain("mixed", toks)
    rows = [s.feed([("a", toks[:20], [19])])]
    for t in range(20, 250):
        rows.append(s.feed([("a", toks[t:t + 1], [0])]))
    close_logits(torch.cat(rows), ref[19:], F32)


def test_plain_forms_by_switch(monkeypatch):
    """QSPEC_SEQ_TILES=0: no tensor-core form of attention, experts or recurrences; the logits stay those of the tile forms."""
    toks = tokens(100, 97, 9)
    cfg, w, model, s = build("wide", BF16, max_step_tokens=128)
    assert model.use_tiles
    tiles = s.feed([("a", toks, list(range(100)))]).float().cpu()
    monkeypatch.setenv("QSPEC_SEQ_TILES", "0")
    cfg, w, model, s = build("wide", BF16, max_step_tokens=128)
    assert not model.use_tiles
    close_logits(s.feed([("a", toks, list(range(100)))]), tiles, BF16, same_format=True)


def test_greedy_generation_through_the_scheduler():
    cfg, w, model, s = build("mixed", F32, n_slots=2, max_step_tokens=16)
    prompts = [tokens(9, cfg["vocab"], 31), tokens(21, cfg["vocab"], 32), tokens(3, cfg["vocab"], 33)]
    outs = s.generate(prompts, 6)
    for p, o in zip(prompts, outs):
        seq = list(p)
        for t in o:
            lg = O.forward(cfg, w, seq)[-1]
            top2 = torch.topk(lg, 2).values
            if float(top2[0] - top2[1]) > 1e-3 * float(lg.abs().max()):     # a near tie may fall either way
                assert int(torch.argmax(lg)) == t
            seq.append(t)


def test_checkpoint_folder_through_the_registry_the_command_line_and_the_trace_replay(tmp_path, capsys):
    """config.json + model.safetensors -> registry -> the `generate` command and the replay program's main()."""
    _cuda()
    import io
    import sys
    import numpy as np
    from qspec_b200 import registry
    from qspec_b200.__main__ import main as cli
    from qspec_b200.checkpoint import write_safetensors_file
    from qspec_b200.totatar import TotatarConfig, random_weights
    from qspec_b200.trace import main
    cfg = CONFIGS["odd"]
    w = random_weights(TotatarConfig.from_dict(cfg), 0)
    with open(tmp_path / "config.json", "w") as f:
        json.dump(cfg, f)
    write_safetensors_file(str(tmp_path / "model.safetensors"), w)
    assert type(registry.load_model(str(tmp_path), dtype="float32", n_slots=1, max_step_tokens=8)).__name__ == "TotatarModel"
    assert cli(["generate", "--model", str(tmp_path), "--dtype", "float32", "--prompt", "5,17,3", "--max-new-tokens", "2"]) == 0
    line = json.loads(capsys.readouterr().out.strip().splitlines()[-1])
    assert line["prompt"] == [5, 17, 3] and len(line["tokens"]) == 2
    assert line["tokens"][0] == int(torch.argmax(O.forward(cfg, w, [5, 17, 3])[-1]))
    toks = tokens(24, cfg["vocab"], 8)
    steps = [{"step": 0, "entries": [{"id": "r", "tokens": toks[:11], "want": [0, 10]}], "end": []},
             {"step": 1, "entries": [{"id": "r", "tokens": toks[11:13], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "r", "tokens": toks[13:], "want": [10]}], "end": ["r"]},
             {"step": 3, "entries": [{"id": "s", "tokens": toks[:2], "want": [1]}], "end": ["s"]}]
    stdin, stdout = sys.stdin, sys.stdout
    sys.stdin, sys.stdout = io.StringIO("\n".join(json.dumps(s) for s in steps) + "\n"), io.StringIO()
    try:
        rc = main(["--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path / "out"), "--max-tokens", "32"])
        printed = sys.stdout.getvalue()
    finally:
        sys.stdin, sys.stdout = stdin, stdout
    assert rc == 0 and [l for l in printed.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
    ref = O.forward(cfg, w, toks)
    assert not os.path.exists(tmp_path / "out" / "1.f32")
    for step, rows in ((0, [0, 10]), (2, [23]), (3, [1])):
        got = torch.from_numpy(np.fromfile(tmp_path / "out" / f"{step}.f32", dtype="<f4").reshape(len(rows), cfg["vocab"]))
        close_logits(got, ref[rows], F32)
