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
                                                    (4, 1, 96, 40, True, 1), (2, 1, 160, 90, True, 0), (1, 1, 300, 6, False, 0)])
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
@pytest.mark.parametrize("H,G,D,DV,taps,every", [(4, 2, 16, 24, 3, 5), (3, 3, 10, 6, 4, 0), (2, 1, 7, 33, 1, 3), (4, 4, 48, 96, 2, 256), (2, 1, 130, 8, 5, 7),
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


FORMS = [("plain", F32, (4, 2, 16, 24)), ("plain", BF16, (4, 2, 16, 24)), ("plain", F32, (3, 1, 33, 7)), ("plain", BF16, (2, 2, 96, 96)),
         ("plain", F32, (2, 1, 48, 130)), ("heads", BF16, (4, 2, 64, 64)), ("heads", BF16, (8, 1, 128, 128)), ("rows", BF16, (4, 2, 64, 128)),
         ("rows", BF16, (2, 2, 128, 64)), ("tile", BF16, (2, 1, 64, 64)), ("tile", BF16, (4, 2, 128, 128))]


@pytest.mark.parametrize("form,dtype,sizes", FORMS)
@pytest.mark.parametrize("window,keep", [(40, 4), (72, 1), (17, 20), (FULL, 0), (1, 3), (64, 0)])
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
