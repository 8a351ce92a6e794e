"""Legavik on the GPU against the plain CPU restatement (oracle/legavik_oracle.py): every mechanism alone, then whole models through the
scheduler's step function -- whole prompts, token-by-token decoding, portions down to two tokens, mixed batches, reused slots, windows
and kept first tokens at their edges, far keys, other sizes, long decoding and greedy generation."""
import json
import math
import os

import pytest
import torch

from oracle import legavik_oracle as O

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


def close(got, want, dtype, scale=None):
    want = want.to(F64)
    s = float(want.abs().max()) if scale is None else scale
    err = float((got.detach().cpu().to(F64) - want).abs().max())
    assert err <= tol(dtype) * max(s, 1e-6), f"max error {err:.3g} against scale {s:.3g}"


def dev(t, dtype=F32):
    return t.to(dtype).cuda().contiguous()


# ---------------------------------------------------------------------------------------------------------------------
# mechanisms alone
# ---------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("W", [96, 257, 40, 2052])
def test_residual_sum_and_tanh_norm(dtype, W):
    """One part with a bias per column; several weighted parts; no sublayer at all. Values far out saturate the tanh."""
    _cuda()
    from qspec_b200 import ops
    g = torch.Generator().manual_seed(W)
    T, alpha = 7, 0.7
    x, y, w, b, bias = rnd(g, T, W, scale=3.0), rnd(g, T, W, dtype=dtype), rnd(g, W), rnd(g, W), rnd(g, W)
    x[0, 0], x[1, 1] = 500.0, -500.0
    sd = {"n": w, "n.b": b, "n.alpha": torch.tensor(alpha)}
    xo, out = torch.empty(T, W, dtype=F32, device="cuda"), torch.empty(T, W, dtype=dtype, device="cuda")
    ops.seq_residual_tanh(dev(x), alpha, dev(w), dev(b), y=dev(y, dtype), y_bias=dev(bias), mult=0.5, x_out=xo, out=out)
    r = x + 0.5 * (y + bias)
    close(xo, r, F32)
    close(out, torch.tanh(alpha * r) * w + b, dtype)
    parts, wt = rnd(g, T, 3, W, dtype=dtype), rnd(g, T, 3)
    xi = dev(x)
    ops.seq_residual_tanh(xi, alpha, dev(w), dev(b), y=dev(parts, dtype), y_w=dev(wt), x_out=xi, out=out)
    r = x + (parts * wt[:, :, None]).sum(1)
    close(xi, r, F32)
    close(out, torch.tanh(alpha * r) * w + b, dtype)
    ops.seq_residual_tanh(dev(x), alpha, dev(w), dev(b), out=out)
    close(out, O.tanh_norm(x, {**sd, "n.alpha": torch.tensor(alpha, dtype=F64)}, "n"), dtype)


def test_logit_soft_cap():
    _cuda()
    from qspec_b200 import ops
    g = torch.Generator().manual_seed(1)
    for shape in ((3, 41), (5, 64), (1, 1)):
        z = rnd(g, *shape, scale=20.0)
        a = dev(z)
        ops.seq_softcap(a, 12.5)
        close(a, O.softcap(z, 12.5), F32)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("E,top,groups,keep", [(6, 2, 3, 2), (12, 4, 2, 1), (8, 3, 1, 1), (9, 9, 3, 3), (40, 5, 8, 2), (5, 1, 5, 1)])
def test_softmax_router_with_groups_and_normalised_weights(dtype, E, top, groups, keep):
    _cuda()
    from qspec_b200 import ops
    g = torch.Generator().manual_seed(E * 10 + top)
    T, W = 23, 36
    h, rw = rnd(g, T, W, dtype=dtype), rnd(g, E, W, scale=0.6)
    idx, wt = torch.empty(T, top, dtype=torch.int32, device="cuda"), torch.empty(T, top, dtype=F32, device="cuda")
    ops.moe_route_grouped(dev(h, dtype), dev(rw), None, idx, wt, score="softmax", groups=groups, keep=keep, group_top=1, normalize=True)
    for t in range(T):
        want = O.route(rw @ h[t], top, groups, keep)
        assert idx[t].tolist() == [e for e, _ in want]
        close(wt[t], torch.tensor([p for _, p in want], dtype=F64), F32)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("H,G,D,dims,scaled,keep", [(4, 2, 16, 12, True, 0), (3, 1, 10, 4, False, 2), (2, 2, 7, 0, False, 0), (6, 2, 64, 64, True, 3),
                                                    (4, 1, 112, 40, True, 1), (2, 1, 160, 90, True, 0), (1, 1, 300, 6, False, 0)])
def test_window_heads_rotation_then_unit_norm_values_are_the_projected_keys(dtype, H, G, D, dims, scaled, keep):
    """Cache rows of a ring with pinned first rows: the step crosses the ring's end, two sequences share it."""
    _cuda()
    from qspec_b200 import ops
    g = torch.Generator().manual_seed(H * 100 + D)
    eps, cap = 1e-5, 13                                                  # the longest run of a step fits the rows that turn over
    segs = [(2, 9, 9), (0, 0, 3), (1, 40, 1)]
    T = sum(s[2] for s in segs)
    sc = {"factor": 4.0, "original": 128, "fast": 16.0, "slow": 1.0} if scaled else None
    p = rnd(g, T, (H + G) * D + H + 3, dtype=dtype)
    pos = torch.tensor([p0 + i for _, p0, n in segs for i in range(n)])
    fr, amp = (O.yarn_frequencies(dims, 60.0, sc), O.yarn_amplitude(sc)) if dims else ([], 1.0)
    q, k = p[:, :H * D].reshape(T, H, D), p[:, H * D:(H + G) * D].reshape(T, G, D)
    v = k.clone()
    q, k = O.unit_rms(O.rotate_halves(q, pos, fr, amp), eps), O.unit_rms(O.rotate_halves(k, pos, fr, amp), eps)
    ck = torch.full((4, cap, G, D), 9.0, dtype=dtype, device="cuda")
    cv = torch.full((4, cap, G, D), 9.0, dtype=dtype, device="cuda")
    qo = torch.empty(T, H, D, dtype=F32, device="cuda")
    meta = plan(segs)
    ops.seq_head_prep(dev(p, dtype), 0, H * D, None, qo, ck, cv, meta.table, H, eps, norm_last=True, inv_freq=dev(torch.tensor(fr)) if dims else None,
                      rot_dims=dims, rot_amp=amp, keep_first=keep)
    close(qo, q, F32)
    at, touched = 0, set()
    for slot, p0, n in segs:
        for i in range(n):
            j = p0 + i
            row = j if j < cap else keep + (j - keep) % (cap - keep)
            close(ck[slot, row], k[at], dtype)
            close(cv[slot, row], v[at], dtype)
            touched.add((slot, row))
            at += 1
    for slot in range(4):
        for row in range(cap):
            if (slot, row) not in touched:
                assert float((ck[slot, row] - 9.0).abs().max()) == 0.0


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("H,G,D,DV,taps,every", [(4, 2, 16, 24, 3, 5), (3, 3, 10, 6, 4, 0), (2, 1, 7, 33, 1, 3), (4, 4, 40, 88, 2, 128), (2, 1, 130, 8, 5, 7),
                                                 (6, 2, 64, 64, 4, 1)])
def test_convolved_heads_with_norm_and_temperature_over_portions(dtype, H, G, D, DV, taps, every):
    """Portions shorter than the convolution, another sequence in between, a new sequence in a used slot."""
    _cuda()
    from qspec_b200 import ops
    g = torch.Generator().manual_seed(D * 10 + taps)
    eps, T, cap, coef = 1e-5, 37, 64, 0.4
    C = H * D + G * D + G * DV
    x, w = rnd(g, T, C, dtype=dtype), rnd(g, C, taps)
    qn, kn = rnd(g, D, scale=0.2) + 1.0, rnd(g, D, scale=0.2) + 1.0
    y = O.causal_conv(x, w)
    q = O.unit_rms(y[:, :H * D].reshape(T, H, D), eps) * qn
    k = O.unit_rms(y[:, H * D:(H + G) * D].reshape(T, G, D), eps) * kn
    v = y[:, (H + G) * D:].reshape(T, G, DV)
    if every:
        q = q * O.temperature(torch.arange(T), coef, every)[:, None, None]
    tail = torch.full((2, 4, taps - 1, C), 7.0, dtype=F32, device="cuda")
    ck, cv = (torch.zeros(4, cap, G, n, dtype=dtype, device="cuda") for n in (D, DV))
    wd = dev(w.t())
    pad = torch.cat([x, torch.full((T, 5), 3.0, dtype=F64)], 1)

    def step(segs):
        meta = plan(segs)
        rows = torch.cat([pad[p0:p0 + n] for _, p0, n, _ in segs])
        qo = torch.empty(rows.shape[0], H, D, dtype=F32, device="cuda")
        ops.seq_head_prep(dev(rows, dtype), 0, H * D, (H + G) * D, qo, ck, cv, meta.table, H, eps, conv_w=wd, tail=tail, qn_w=dev(qn), kn_w=dev(kn),
                          temp_coef=coef, temp_every=every)
        at = 0
        for slot, p0, n, _ in segs:
            close(qo[at:at + n], q[p0:p0 + n], F32, scale=float(q.abs().max()))
            close(ck[slot, p0:p0 + n], k[p0:p0 + n], dtype, scale=float(k.abs().max()))
            close(cv[slot, p0:p0 + n], v[p0:p0 + n], dtype, scale=float(v.abs().max()))
            at += n

    step([(1, 0, T, 0)])
    at, ph = 0, 1                                                         # slot 1 again from its start, its phase as the last step left it
    for n in (1, 1, 2, 1, 9, 2, 3, 18):
        step([(1, at, n, ph), (3, 0, 4, 0)])
        at += n
        ph ^= 1


class DeltaCase:
    """Inputs of the delta rule for several sequences, the plain result, and a step function over (slot, first, count, phase, sequence)."""

    def __init__(self, dtype, H, G, D, DV, taps, T, seed, nseq=2, strong=False):
        g = torch.Generator().manual_seed(seed)
        self.dtype, self.dims, self.eps = dtype, (H, G, D, DV), 1e-5
        C = 2 * G * D + H * DV
        self.x = [rnd(g, T, C, dtype=dtype) for _ in range(nseq)]
        self.beta = [rnd(g, T, H, dtype=dtype, scale=2.0) for _ in range(nseq)]
        self.a = [rnd(g, T, H * D, scale=6.0 if strong else 1.5) for _ in range(nseq)]
        self.gate = [rnd(g, T, H * DV, dtype=dtype) for _ in range(nseq)]
        self.w = rnd(g, C, taps, scale=0.6)
        self.A_log, self.dt_bias = rnd(g, H, scale=0.5), rnd(g, H * D, scale=0.5) - 1.0
        if strong:
            self.A_log = self.A_log + 2.0                              # decays of e^-30 a token and more next to hardly any
        self.norm = rnd(g, DV, scale=0.1) + 1.0
        self.state = torch.full((4, H, D, DV), 3.0, dtype=F32, device="cuda")
        self.tail = torch.full((2, 4, taps - 1, C), 7.0, dtype=F32, device="cuda")
        self.want = [self._plain(i) for i in range(nseq)]

    def _plain(self, i):
        H, G, D, DV = self.dims
        T = self.x[i].shape[0]
        y = O.silu(O.causal_conv(self.x[i], self.w))
        q, k, v = y[:, :G * D].reshape(T, G, D), y[:, G * D:2 * G * D].reshape(T, G, D), y[:, 2 * G * D:].reshape(T, H, DV)
        q = q / torch.sqrt((q * q).sum(-1, keepdim=True) + 1e-6) / math.sqrt(D)
        k = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
        dec = torch.exp(-torch.exp(self.A_log)[None, :, None] * O.softplus(self.a[i] + self.dt_bias).view(T, H, D))
        o = O.delta_rule(q, k, v, torch.sigmoid(self.beta[i]), dec)
        return (O.unit_rms(o, self.eps) * self.norm * torch.sigmoid(self.gate[i]).view(T, H, DV)).reshape(T, H * DV) * 1.25

    def step(self, segs):
        from qspec_b200 import ops
        H, G, D, DV = self.dims
        meta = plan([s[:4] for s in segs])
        cat = lambda per: torch.cat([per[i][p0:p0 + n] for _, p0, n, _, i in segs])
        p = torch.cat([cat(self.x), torch.full((meta.ntok, 2), 5.0, dtype=F64), cat(self.beta)], 1)     # two columns of something else between
        wide = torch.full((meta.ntok, H * DV + 4), -1.0, dtype=self.dtype, device="cuda")
        out = wide[:, 4:]
        nb = meta.block_rows.numel()
        scratch = torch.full((max(ops.seq_delta_channel_scratch_bytes(nb, meta.ntok, H, D, DV), 16),), 255, dtype=torch.uint8, device="cuda")
        ops.seq_delta_channel(dev(p, self.dtype), self.x[0].shape[1] + 2, dev(self.w.t()), self.tail, dev(cat(self.a)), dev(self.A_log),
                              dev(self.dt_bias), dev(self.norm), dev(cat(self.gate), self.dtype), self.state, out, meta, G, self.eps,
                              scratch=scratch, out_scale=1.25)
        assert float((wide[:, :4] + 1.0).abs().max()) == 0.0
        at = 0
        for _, p0, n, _, i in segs:
            close(out[at:at + n], self.want[i][p0:p0 + n], self.dtype, scale=float(self.want[i].abs().max()))
            at += n


DELTA_SIZES = [(2, 2, 16, 24, 4), (4, 2, 33, 7, 2), (3, 1, 130, 40, 3), (2, 2, 64, 64, 1), (6, 3, 5, 17, 6), (1, 1, 200, 16, 4), (2, 1, 128, 128, 4),
               (1, 1, 12, 300, 3), (2, 1, 256, 20, 2)]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("H,G,D,DV,taps", DELTA_SIZES)
def test_delta_rule_with_channel_decays_over_portions_and_slots(dtype, H, G, D, DV, taps):
    """Both forms: the whole sequence at once (blocks), then portions from one token to more than two blocks with another sequence
    stepping through a neighbouring slot -- token form and block form in one step, segments that end inside a block --, from
    position 0 in a used slot."""
    _cuda()
    c = DeltaCase(dtype, H, G, D, DV, taps, T=75, seed=H * 1000 + D)
    c.step([(1, 0, 75, 0, 0)])
    at, ph = 0, 1
    for n in (1, 2, 8, 9, 1, 16, 3, 17, 18):
        c.step([(1, at, n, ph, 0), (0, 0, min(at, 40) + 1, 0, 1)])         # the second sequence restarts in every step, longer and longer
        at += n
        ph ^= 1
    assert at == 75


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_delta_rule_with_decays_that_empty_a_channel_within_a_token(dtype):
    """Decays from nearly one down to far below the smallest float32 number: their ratios inside a block must not overflow."""
    _cuda()
    c = DeltaCase(dtype, 2, 1, 40, 20, 3, T=50, seed=9, strong=True)
    c.step([(2, 0, 50, 0, 0)])
    for t in range(12):
        c.step([(3, t, 1, t & 1, 1)])


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_delta_rule_tokens_one_by_one_equal_the_blocks(dtype):
    _cuda()
    c = DeltaCase(dtype, 2, 2, 24, 16, 4, T=40, seed=3)
    for t in range(40):
        c.step([(0, t, 1, t & 1, 0), (2, t, 1, t & 1, 1)])


# ---- attention with a window and kept first tokens: the plain form and the tensor-core forms ----
def _ring(k, slot, slots, cap, keep, dtype):
    """Rows of positions 0 .. n - 1 as steps would leave them in a ring of cap rows (later positions overwrite earlier ones)."""
    c = torch.full((slots, cap) + tuple(k.shape[1:]), 9.0, dtype=dtype, device="cuda")
    for j in range(k.shape[0]):
        c[slot, j if j < cap else keep + (j - keep) % (cap - keep)] = dev(k[j], dtype)
    return c


def _attend(form, q, ck, cv, out, meta, window, scale, **kw):
    from qspec_b200 import ops
    if form == "plain":
        ops.seq_window_attention(q, None, ck, cv, out, meta.table, window, scale, **kw)
    elif form == "tile":
        _, slot, pos0, _ = meta.segments[0]
        ops.seq_prompt_attention_mma(q, ck, None, cv, out, slot, pos0, window, scale, **kw)
    else:
        ops.seq_window_attention_mma(q, ck, None, cv, out, meta.table, window, scale, form == "rows", **kw)


FORMS = [("plain", F32, (4, 2, 16, 24)), ("plain", BF16, (4, 2, 16, 24)), ("plain", F32, (3, 1, 33, 7)), ("plain", BF16, (2, 2, 80, 80)),
         ("plain", F32, (2, 1, 36, 130)), ("heads", BF16, (4, 2, 64, 64)), ("heads", BF16, (8, 1, 128, 128)), ("rows", BF16, (4, 2, 64, 128)),
         ("rows", BF16, (2, 2, 128, 64)), ("tile", BF16, (2, 1, 64, 64)), ("tile", BF16, (4, 2, 128, 128))]


@pytest.mark.parametrize("form,dtype,sizes", FORMS)
@pytest.mark.parametrize("window,keep", [(40, 4), (70, 1), (17, 20), (FULL, 0), (1, 3), (64, 0)])
def test_window_with_kept_first_tokens(form, dtype, sizes, window, keep):
    """A portion late in the sequence, one that starts inside the kept tokens' reach, single tokens; the ring has wrapped several
    times; output columns of a wider buffer, a gate per head and an output factor."""
    _cuda()
    H, G, D, DV = sizes
    g = torch.Generator().manual_seed(H * 100 + D + min(window, 999))
    n = 230
    q, k, v = rnd(g, n, H, D), rnd(g, n, G, D, dtype=dtype), rnd(g, n, G, DV, dtype=dtype)
    gate = rnd(g, n, H, dtype=dtype)
    scale = 0.9 / math.sqrt(D)
    want = O.masked_attention(q, k, v, scale, None if window == FULL else window, keep) * torch.sigmoid(gate)[:, :, None] * 1.25
    top = float(want.abs().max())
    for first, count in ((n - 90, 90), (n - 2, 2), (n - 1, 1), (0, 25), (keep + 1, 70)):
        if form == "tile" and count < 3:
            continue
        end = first + count
        cap = n + 3 if window == FULL else min(n, keep + window - 1 + count + 2)
        ck, cv = _ring(k[:end], 1, 3, cap, keep, dtype), _ring(v[:end], 1, 3, cap, keep, dtype)
        meta = plan([(1, first, count)])
        wide = torch.full((count, H * DV + 8), -1.0, dtype=dtype, device="cuda")
        out = wide.as_strided((count, H, DV), (H * DV + 8, DV, 1), 4)
        _attend(form, dev(q[first:end]), ck, cv, out, meta, window, scale, gate=dev(gate[first:end], dtype), gate_per_head=True, keep_first=keep,
                out_scale=1.25)
        close(out, want[first:end], dtype, scale=top)
        assert float((wide[:, :4] + 1.0).abs().max()) == 0.0 and float((wide[:, -4:] + 1.0).abs().max()) == 0.0
    if form == "tile":
        return
    # two sequences and single tokens in one step
    m = 60
    ck, cv = _ring(k[:n], 1, 3, n, keep, dtype), _ring(v[:n], 1, 3, n, keep, dtype)
    q2, k2, v2 = rnd(g, m, H, D), rnd(g, m, G, D, dtype=dtype), rnd(g, m, G, DV, dtype=dtype)
    ck[2, :m], cv[2, :m] = dev(k2, dtype), dev(v2, dtype)
    want2 = O.masked_attention(q2, k2, v2, scale, None if window == FULL else window, keep)
    meta = plan([(2, 10, 50), (1, n - 5, 5)])
    out = torch.empty(55, H, DV, dtype=dtype, device="cuda")
    _attend(form, dev(torch.cat([q2[10:], q[n - 5:]])), ck, cv, out, meta, window, scale, keep_first=keep)
    close(out[:50], want2[10:], dtype, scale=float(want2.abs().max()))
    plain = want[n - 5:] / (torch.sigmoid(gate[n - 5:])[:, :, None] * 1.25)
    close(out[50:], plain, dtype, scale=float(plain.abs().max()))


@pytest.mark.parametrize("form,dtype,sizes", [("plain", F32, (2, 1, 32, 16)), ("plain", BF16, (2, 1, 32, 16)), ("heads", BF16, (2, 1, 64, 64)),
                                              ("rows", BF16, (2, 1, 64, 64)), ("tile", BF16, (2, 1, 64, 64))])
@pytest.mark.parametrize("place", ["window_in", "window_out", "first_in", "first_out", "far"])
def test_a_key_that_stands_out_at_every_edge(form, dtype, sizes, place):
    """One key matches the last query far better than the hundreds of others and its value stands out: just inside the window or among
    the kept tokens the output carries it; one position further out it does not."""
    _cuda()
    H, G, D, DV = sizes
    g = torch.Generator().manual_seed(17)
    n, window, keep = 420, 100, 4
    q, k, v = rnd(g, n, H, D, scale=0.3), rnd(g, n, G, D, dtype=dtype, scale=0.3), rnd(g, n, G, DV, dtype=dtype, scale=0.1)
    j = {"window_in": n - window, "window_out": n - 1 - window, "first_in": keep - 1, "first_out": keep, "far": 37}[place]
    seen = place in ("window_in", "first_in", "far")
    w, kf = (FULL, 0) if place == "far" else (window, keep)
    k[j, 0] = (q[n - 1, 1] * 8.0).to(dtype).to(F64)
    v[j, 0] = 5.0
    want = O.masked_attention(q, k, v, 1.0, None if w == FULL else w, kf)
    assert (float(want[n - 1, 1].mean()) > 2.0) == seen
    cap = n if w == FULL else keep + window - 1 + 30
    ck, cv = _ring(k, 0, 2, cap, kf, dtype), _ring(v, 0, 2, cap, kf, dtype)
    for count in (30, 1):
        if form == "tile" and count == 1:
            continue
        meta = plan([(0, n - count, count)])
        out = torch.empty(count, H, DV, dtype=dtype, device="cuda")
        _attend(form, dev(q[n - count:]), ck, cv, out, meta, w, 1.0, keep_first=kf)
        close(out, want[n - count:], dtype, scale=float(want[n - count:].abs().max()))
        assert (float(out[-1, 1].float().mean()) > 2.0) == seen


# ---------------------------------------------------------------------------------------------------------------------
# whole models through the scheduler
# ---------------------------------------------------------------------------------------------------------------------
def attention(heads=4, kv_heads=2, dim=16, scale=0.3, window=20, keep=3, dims=None, base=500.0, scaling=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "mask": {"size": window, "keep_first": keep},
         "rot": {"base": base, "dims": dim if dims is None else dims}}
    if scaling:
        m["rot"]["scaling"] = scaling
    return {"type": "attention", "mixer": m}


def parallel(left=(4, 2, 16, 12), lconv=3, temp=(0.3, 8), right=(4, 2, 12, 10), rconv=4, scales=(0.8, 1.25), scale=0.25):
    lh, lg, ld, lv = left
    rh, rg, rd, rv = right
    lm = {"heads": lh, "kv_heads": lg, "dim": ld, "vdim": lv, "conv": lconv, "scale": scale}
    if temp:
        lm["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return {"type": "parallel", "mixer": {"left": lm, "right": {"heads": rh, "kv_heads": rg, "dim": rd, "vdim": rv, "conv": rconv},
                                          "left_scale": scales[0], "right_scale": scales[1]}}


def moe(ff=24, experts=8, top=3, count=4, keep=2):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}}}


def config(layers, width=64, vocab=97, eps=1e-5, softcap=12.0):
    return {"architecture": "Legavik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_softcap": softcap, "layers": layers}


STRETCH = {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}
CONFIGS = {
    # both mixers, grouped heads on every side, windows shorter and longer than the portions
    "mixed": (config([dict(attention(scaling=STRETCH), mlp=moe()), dict(parallel(), mlp=moe(ff=16, experts=6, top=2, count=2, keep=1)),
                      dict(attention(heads=6, kv_heads=1, dim=8, dims=4, window=33, keep=0), mlp=None),
                      dict(parallel(left=(2, 2, 24, 8), right=(6, 3, 8, 6), lconv=2, rconv=2), mlp=moe())]), 5, 7),
    # nothing divisible by anything: one head, all heads on one key, one-tap and long convolutions, no temperature, no rotation, one
    # expert per token, as many chosen as there are, a window of one token, layers that open with a parallel mixer
    "odd": (config([dict(parallel(left=(3, 3, 10, 7), right=(1, 1, 33, 7), lconv=1, rconv=5, temp=None, scales=(1.0, 1.0)), mlp=None),
                    dict(attention(heads=3, kv_heads=1, dim=10, dims=0, window=1, keep=2), mlp=moe(ff=13, experts=5, top=1, count=1, keep=1)),
                    dict(parallel(left=(1, 1, 6, 9), right=(3, 1, 5, 17), lconv=6, rconv=1, temp=(0.5, 1)), mlp=moe(ff=9, experts=3, top=3, count=3, keep=3)),
                    dict(attention(heads=5, kv_heads=5, dim=7, dims=2, base=37.0, window=9, keep=11), mlp=None)],
                   width=50, vocab=33, eps=1e-6, softcap=5.0), 3, 1),
    # head sizes of the tensor-core forms, a key size above 128 in the recurrence, values wider than one pass
    "wide": (config([dict(attention(heads=4, kv_heads=2, dim=64, dims=32, scaling=STRETCH, scale=0.12, window=48, keep=4), mlp=moe(ff=32)),
                     dict(parallel(left=(4, 1, 64, 128), right=(2, 1, 130, 40), scale=0.1), mlp=None),
                     dict(parallel(left=(2, 2, 128, 64), right=(2, 2, 24, 136), scale=0.08), mlp=moe(ff=32))], width=96, softcap=20.0), 16, 8),
}


def build(name, dtype, seed=0, n_slots=3, max_step_tokens=64, max_seq_tokens=256):
    _cuda()
    from qspec_b200.legavik import LegavikConfig, LegavikModel, random_weights
    from qspec_b200.scheduler import Scheduler
    d, rd, rg = CONFIGS[name]
    cfg = LegavikConfig.from_dict(d)
    w = random_weights(cfg.with_ranks(decay_rank=rd, gate_rank=rg), seed)
    model = LegavikModel(cfg, w, dtype=dtype, device="cuda", n_slots=n_slots, max_step_tokens=max_step_tokens, max_seq_tokens=max_seq_tokens)
    model.prompt_tiles_min_ctas = 2                        # short test prompts take the tile form too
    return d, w, model, Scheduler(model)


def tokens(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def close_logits(got, ref, dtype, same_format=False):
    """Per position: root mean square over the vocabulary of the difference (mean taken off), relative to the spread of the
    logits. float32 against the plain implementation: rounding level. bfloat16 against the plain implementation: what an 8-bit
    mantissa leaves, with a few positions further off where two experts' scores are nearly equal. same_format: bfloat16 against
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
        from qspec_b200.legavik import LegavikConfig, random_weights
        d, rd, rg = CONFIGS[name]
        lay = []
        _PLAIN[key] = (O.forward(d, random_weights(LegavikConfig.from_dict(d).with_ranks(decay_rank=rd, gate_rank=rg), seed), toks, lay), lay)
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
    toks = tokens(90, cfg["vocab"], 1)
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
    """Token by token from the first token on; a prompt then 40 single tokens; portions of 2, 3, 1, 7, ... tokens; a step
    longer than the model's step size (cut inside the step function)."""
    cfg, w, model, s = build(name, dtype, max_step_tokens=16)
    toks = tokens(90, cfg["vocab"], 1)
    ref = reference_logits(name, toks, dtype)
    schedules = {"single": [1] * len(toks), "prompt+decode": [16, 16, 16, 2] + [1] * 40, "twos": [2] * 45,
                 "portions": [2, 3, 1, 7, 2, 2, 13, 5, 2, 16, 9, 11, 14, 3], "one step": [len(toks)]}
    for label, cuts in schedules.items():
        assert sum(cuts) == len(toks)
        at, rows = 0, []
        for n in cuts:
            rows.append(s.feed([(label, toks[at:at + n], list(range(n)))]))
            at += n
        s.release(label)
        close_logits(torch.cat(rows), ref, dtype, same_format=True)


@pytest.mark.parametrize("name", ["mixed", "wide"])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_mixed_batches_equal_each_request_alone_and_slots_are_reused(name, dtype):
    """Three requests of unequal length advance together -- a prompt portion next to single tokens next to a request that
    starts late in a slot another request has just given back -- and each must see what it sees alone."""
    cfg, w, model, s = build(name, dtype, n_slots=2, max_step_tokens=48)
    seqs = {"a": tokens(60, cfg["vocab"], 11), "b": tokens(23, cfg["vocab"], 12), "c": tokens(41, cfg["vocab"], 13)}
    alone = {}
    for rid, toks in seqs.items():
        alone[rid] = s.feed([(rid, toks, list(range(len(toks))))]).float().cpu()
        s.release(rid)
        if dtype == F32:
            close_logits(alone[rid], plain(name, toks), dtype)
    sched = [{"a": 7, "b": 20}, {"a": 1, "b": 1}, {"a": 30, "b": 2}, {"a": 1}, {"a": 1, "c": 9}, {"a": 2, "c": 1}, {"a": 18, "c": 30}, {"c": 1}]
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
    bias included."""
    from qspec_b200.legavik import LegavikConfig, LegavikModel, random_weights
    from qspec_b200.scheduler import Scheduler
    _cuda()
    scales = (1.5, 0.0) if half == "left" else (0.0, 1.5)
    d = config([dict(parallel(scales=scales), mlp=None), dict(parallel(scales=scales), mlp=moe())])
    w = random_weights(LegavikConfig.from_dict(d).with_ranks(decay_rank=5, gate_rank=7), 4)
    toks = tokens(40, 97, 4)
    ref = O.forward(d, w, toks)
    other = "right" if half == "left" else "left"
    w2 = {k: (v.flip(0) * 2.0 if f".{other}." in k and v.dim() else v) for k, v in w.items()}
    for ww in (w, w2):
        m = LegavikModel(LegavikConfig.from_dict(d), ww, dtype=F32, device="cuda", n_slots=1, max_step_tokens=20, max_seq_tokens=64)
        close_logits(Scheduler(m).feed([("a", toks, list(range(40)))]), ref, F32)


def test_the_ring_of_a_window_layer_is_short_and_keeps_its_first_rows():
    """A model of window layers alone does not bound the sequence: its rings hold the kept rows, the window and a step; far beyond
    them, prompts and decoding still equal the plain implementation."""
    from qspec_b200.legavik import LegavikConfig, LegavikModel, random_weights
    from qspec_b200.scheduler import Scheduler
    _cuda()
    d = config([dict(attention(window=12, keep=3, scaling=STRETCH), mlp=None), dict(attention(window=5, keep=6, heads=2, kv_heads=2), mlp=moe())])
    w = random_weights(LegavikConfig.from_dict(d), 6)
    m = LegavikModel(LegavikConfig.from_dict(d), w, dtype=F32, device="cuda", n_slots=2, max_step_tokens=10)
    assert m.max_seq_len is None and m.cache_k[0].shape[1] == 3 + 12 - 1 + 10 and m.cache_k[1].shape[1] == 6 + 5 - 1 + 10
    s = Scheduler(m)
    toks = tokens(160, 97, 7)
    ref = O.forward(d, w, toks)
    for label, cuts in (("whole", [160]), ("decode", [70] + [1] * 90), ("portions", [10, 2, 3, 10, 7] * 5)):
        at, rows = 0, []
        for n in cuts:
            rows.append(s.feed([(label, toks[at:at + n], list(range(n)))]))
            at += n
        close_logits(torch.cat(rows), ref, F32)
        s.release(label)


def test_the_cache_bounds_the_sequence_and_the_scheduler_refuses_more():
    cfg, w, model, s = build("mixed", BF16, max_seq_tokens=40)
    s.feed([("a", tokens(40, cfg["vocab"], 5), [39])])
    with pytest.raises(RuntimeError):
        s.feed([("a", [1], [0])])


def test_long_decoding():
    """A short prompt, then 230 single tokens: windows pass over decoded tokens several times, the recurrences' states and the growing
    cache, against the plain implementation."""
    cfg, w, model, s = build("mixed", F32, max_step_tokens=8, max_seq_tokens=512)
    toks = tokens(250, cfg["vocab"], 6)
    ref = plain("mixed", toks)
    rows = [s.feed([("a", toks[:20], [19])])]
    for t in range(20, 250):
        rows.append(s.feed([("a", toks[t:t + 1], [0])]))
    close_logits(torch.cat(rows), ref[19:], F32)


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
    from qspec_b200.legavik import LegavikConfig, random_weights
    from qspec_b200.trace import main
    cfg, rd, rg = CONFIGS["odd"]
    w = random_weights(LegavikConfig.from_dict(cfg).with_ranks(decay_rank=rd, gate_rank=rg), 3)
    with open(tmp_path / "config.json", "w") as f:
        json.dump(cfg, f)
    write_safetensors_file(str(tmp_path / "model.safetensors"), w)
    assert type(registry.load_model(str(tmp_path), dtype="float32", n_slots=1, max_step_tokens=8, max_seq_tokens=32)).__name__ == "LegavikModel"
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
