"""Host-side logic of the Totatar design (no GPU): configuration parsing and tensor names, registry entry, the number formats the
replay program accepts, the chunk tables of a step, and properties of the plain implementation that the GPU tests lean on."""
import json
import math

import pytest
import torch

from oracle import totatar_oracle as O
from qspec_b200 import registry
from qspec_b200.state import CHUNK, CHUNK_MIN, SequenceTable
from qspec_b200.totatar import SECTION, TotatarConfig, _LayerWeights, _sections, random_weights

F64 = torch.float64

MOE = {"kind": "moe", "expert": {"ff": 10}, "router": {"experts": 6, "top": 2}, "shared": {"ff": 7}}
PAR = {"type": "parallel", "mlp": {"kind": "dense", "ff": 11},
       "mixer": {"left": {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 5, "scale": 0.4, "mask": {"size": 5},
                          "rot": {"base": 100.0, "dims": 4, "scaling": {"factor": 2.0}}},
                 "right": {"heads": 3, "dim": 7, "vdim": 9, "decay": [0.5, 0.9, 1.0]}, "left_scale": 0.75, "right_scale": 1.5}}
SSM = {"type": "mamba2", "mlp": MOE, "mixer": {"heads": 4, "groups": 2, "state": 3, "vdim": 5, "conv": 3, "norm_groups": 10}}


def _cfg(layers, width=32, vocab=41):
    return {"architecture": "Totatar", "vocab": vocab, "width": width, "norm": {"eps": 1e-5}, "layers": layers}


def test_configuration_round_trip_and_tensor_names():
    d = _cfg([PAR, SSM, dict(SSM, mlp=None), dict(PAR, mlp=dict(MOE, shared=None))])
    cfg = TotatarConfig.from_dict(d)
    assert TotatarConfig.from_dict(cfg.to_dict()) == cfg
    s = cfg.tensor_shapes()
    assert s["embed"] == (41, 32) and "head" not in s and s["final.norm"] == (32,)
    assert all(s[f"l0.{n}"] == (32,) for n in ("norm1", "norm1b", "norm2", "norm2b")) and "l2.norm2" not in s and "l2.norm1b" in s
    L, R, M = "l0.mix.left.", "l0.mix.right.", "l1.mix."
    assert s[L + "q"] == (24, 32) and s[L + "k.b"] == (12,) and s[L + "v"] == (10, 32) and s[L + "sink"] == (4,) and s[L + "o"] == (32, 20)
    assert s[R + "q"] == (21, 32) and s[R + "v"] == (27, 32) and s[R + "g"] == (27, 32) and s[R + "norm"] == (27,) and s[R + "o"] == (32, 27)
    assert s[M + "in"] == (20 + 20 + 12 + 4, 32) and s[M + "conv"] == (32, 3) and s[M + "conv.b"] == (32,) and s[M + "norm"] == (20,)
    assert all(s[M + n] == (4,) for n in ("dt_bias", "A_log", "D")) and s[M + "o"] == (32, 20)
    assert s["l0.mlp.gate"] == (11, 32) and s["l0.mlp.down"] == (32, 11)
    assert s["l1.mlp.router"] == (6, 32) and s["l1.mlp.router.b"] == (6,) and s["l1.mlp.e5.up"] == (10, 32) and s["l1.mlp.shared.down"] == (32, 7)
    assert "l3.mlp.shared.gate" not in s and set(random_weights(cfg)) == set(s)
    # optional keys: no mask, no rotation, no stretch, key heads and value size by default, one norm group, scales of one
    bare = {"type": "parallel", "mixer": {"left": {"heads": 3, "dim": 4, "scale": 0.5}, "right": {"heads": 1, "dim": 2, "decay": [0.5]}}}
    c2 = TotatarConfig.from_dict(_cfg([bare, {"type": "mamba2", "mixer": {"heads": 2, "state": 3, "vdim": 4, "conv": 1}}]))
    a, m = c2.layers[0].mixer.att, c2.layers[0].mixer
    assert (a.kv_heads, a.vdim, a.rot_dims, a.window, a.rot_factor, m.lin.vdim, m.left_scale, m.right_scale) == (3, 4, 0, None, 1.0, 2, 1.0, 1.0)
    assert c2.layers[1].mixer.ssm.norm_groups == 1 and c2.layers[1].mixer.ssm.groups == 1 and c2.layers[0].mlp is None


@pytest.mark.parametrize("change", [
    lambda d: d["layers"][0].update(type="conv"),
    lambda d: d["layers"][0]["mixer"]["left"].update(kv_heads=3),
    lambda d: d["layers"][0]["mixer"]["left"]["rot"].update(dims=8),
    lambda d: d["layers"][0]["mixer"]["left"]["rot"].update(dims=3),
    lambda d: d["layers"][0]["mixer"]["right"].update(decay=[0.5]),
    lambda d: d["layers"][0]["mixer"]["right"].update(decay=[0.5, 1.5, 0.1]),
    lambda d: d["layers"][0]["mlp"].update(kind="sparse"),
    lambda d: d["layers"][1]["mixer"].update(groups=3),
    lambda d: d["layers"][1]["mixer"].update(norm_groups=3),
    lambda d: d["layers"][1]["mixer"].update(conv=0),
    lambda d: d["layers"][1]["mlp"]["router"].update(top=7),
])
def test_configuration_errors(change):
    d = json.loads(json.dumps(_cfg([PAR, SSM])))
    change(d)
    with pytest.raises(ValueError):
        TotatarConfig.from_dict(d)


def test_registry_and_number_formats(tmp_path):
    assert "Totatar" in registry.architectures()
    assert registry.supports_dtype("Totatar", "bfloat16") and registry.supports_dtype("Totatar", "float32")
    assert not registry.supports_dtype("Totatar", "float16")
    with open(tmp_path / "config.json", "w") as f:
        json.dump(_cfg([PAR]), f)
    from qspec_b200.trace import main
    assert main(["--model", str(tmp_path), "--dtype", "float16", "--out", str(tmp_path / "o")]) == 3


def test_chunk_tables_of_a_step():
    """Segments longer than CHUNK_MIN tokens are cut into chunks of CHUNK from their own first row; short ones have none."""
    t = SequenceTable(8, "cpu", 512)
    lens = [1, CHUNK_MIN + 1, CHUNK_MIN, 2 * CHUNK, 9, CHUNK + 1]
    meta = t.plan([(k, n) for k, n in enumerate(lens)])
    begin, rows, starts, first = 0, [], [], []
    for n in lens:
        if n > CHUNK_MIN:
            starts.append(begin)
            first.append(len(rows))
            rows += list(range(begin, begin + n, CHUNK))
        begin += n
    assert meta.chunk_rows.tolist() == rows and meta.chunk_starts.tolist() == starts and meta.chunk_first.tolist() == first
    assert len(rows) <= sum(lens) // CHUNK_MIN                           # what the model reserves scratch for
    meta = t.plan([("x", 3)])
    assert meta.chunk_rows.numel() == meta.chunk_starts.numel() == 0
    for n in range(CHUNK_MIN + 1, 500):
        assert -(-n // CHUNK) <= n / CHUNK_MIN


def test_fused_rows_start_on_boundaries_and_hold_the_tensors():
    assert _sections([24, 12, 10, 21]) == ([0, 24, 40, 56], 80) and all(o % SECTION == 0 for o in _sections([3, 5, 9, 1])[0])
    cfg = TotatarConfig.from_dict(_cfg([PAR, SSM]))
    w = random_weights(cfg, 2)
    p, m = _LayerWeights(cfg, 0, w, torch.float32, "cpu"), _LayerWeights(cfg, 1, w, torch.float32, "cpu")
    f = lambda n: w[n].float()
    for name, at in (("left.q", p.q), ("left.k", p.k), ("left.v", p.v), ("right.q", p.rq), ("right.k", p.rk), ("right.v", p.rv), ("right.g", p.rg)):
        t = f("l0.mix." + name)
        assert at % SECTION == 0 and torch.equal(p.w_in[at:at + t.shape[0]], t)
    for name, at in (("q.b", p.q), ("k.b", p.k), ("v.b", p.v)):
        t = f("l0.mix.left." + name)
        assert torch.equal(p.b_in[at:at + t.shape[0]], t)
    assert float(p.b_in[p.rq:].abs().max()) == 0.0
    assert torch.equal(p.o[:, :20], f("l0.mix.left.o")) and torch.equal(p.o[:, p.o_right:p.o_right + 27], f("l0.mix.right.o"))
    assert p.log_decay.tolist() == pytest.approx([math.log(0.5), math.log(0.9), 0.0])
    h = torch.randn(3, 32, dtype=torch.float32, generator=torch.Generator().manual_seed(0))
    row, whole = h @ m.w_in.T, h @ f("l1.mix.in").T
    for at, lo, n in ((m.z, 0, 20), (m.x, 20, 20), (m.B, 40, 6), (m.C, 46, 6), (m.dt, 52, 4)):
        assert torch.allclose(row[:, at:at + n], whole[:, lo:lo + n], atol=1e-6)
    for at, lo, n in ((m.x, 0, 20), (m.B, 20, 6), (m.C, 26, 6)):
        assert torch.equal(m.conv[at - m.x:at - m.x + n], f("l1.mix.conv")[lo:lo + n]) and torch.equal(m.conv_b[at - m.x:at - m.x + n],
                                                                                                      f("l1.mix.conv.b")[lo:lo + n])


def test_plain_scalar_decay_reads_what_was_written():
    """A value written along one axis is read back n steps later times the decays since, and a cut carries the state over."""
    T, D, DV = 6, 3, 2
    a = torch.rand(T, 1, generator=torch.Generator().manual_seed(0), dtype=F64)
    k, q, v = torch.zeros(T, 1, D, dtype=F64), torch.zeros(T, 1, D, dtype=F64), torch.zeros(T, 1, DV, dtype=F64)
    k[0, 0, 1], k[1:, 0, 2], q[:, 0, 1] = 1.0, 1.0, 1.0
    v[0, 0] = torch.tensor([2.0, -1.0], dtype=F64)
    o = O.scalar_decay(q, k, v, a)
    keep = 1.0
    for t in range(T):
        keep = keep * float(a[t, 0]) if t else 1.0
        assert torch.allclose(o[t, 0], v[0, 0] * keep, atol=1e-14)
    gen = torch.Generator().manual_seed(1)
    q, k = torch.randn(6, 2, D, generator=gen, dtype=F64), torch.randn(6, 2, D, generator=gen, dtype=F64)
    v, a = torch.randn(6, 4, DV, generator=gen, dtype=F64), torch.rand(6, 4, generator=gen, dtype=F64)
    S = torch.zeros(4, D, DV, dtype=F64)
    parts = torch.cat([O.scalar_decay(q[x:y], k[x:y], v[x:y], a[x:y], S) for x, y in ((0, 4), (4, 6))])
    assert torch.allclose(O.scalar_decay(q, k, v, a), parts, atol=1e-12)
    # heads of a group share their keys
    one = O.scalar_decay(q[:, :1], k[:, :1], v[:, :2], a[:, :2])
    assert torch.allclose(O.scalar_decay(q, k, v, a)[:, :2], one, atol=1e-12)


def test_plain_sink_and_window():
    n = 7
    q, k, v = torch.zeros(n, 1, 2, dtype=F64), torch.zeros(n, 1, 2, dtype=F64), torch.eye(n, dtype=F64)[:, None, :]
    o = O.sink_attention(q, k, v, 1.0, 3, torch.tensor([math.log(2.0)], dtype=F64))      # equal scores: 3 keys and a sink of weight 2
    assert torch.allclose(o[5, 0], torch.tensor([0, 0, 0, 1, 1, 1, 0], dtype=F64) / 5.0)
    assert torch.allclose(o[0, 0, 0], torch.tensor(1.0 / 3.0, dtype=F64))
    assert torch.allclose(O.sink_attention(q, k, v, 1.0, None, None)[6, 0], torch.full((n,), 1.0 / n, dtype=F64))


def test_plain_rotation_depends_on_the_distance_alone_and_is_stretched():
    gen = torch.Generator().manual_seed(3)
    x, y = torch.randn(1, 1, 8, generator=gen, dtype=F64), torch.randn(1, 1, 8, generator=gen, dtype=F64)
    fr = O.frequencies(6, 50.0, 2.0)
    at = lambda v, p, f=fr: O.rotate_interleaved(v, torch.tensor([p]), f)
    dots = [float((at(x, p + 5) * at(y, p)).sum()) for p in (0, 9, 200)]
    assert dots[1] == pytest.approx(dots[0]) and dots[2] == pytest.approx(dots[0])
    assert torch.equal(at(x, 7)[..., 6:], x[..., 6:]) and fr[0] == 0.5
    assert torch.allclose(at(x, 10), at(x, 5, O.frequencies(6, 50.0)))
    u = at(torch.eye(8, dtype=F64)[None, :1, :], 1)            # entry 0 turns into entry 1
    assert float(u[0, 0, 1]) == pytest.approx(math.sin(0.5)) and float(u[0, 0, 3:].abs().max()) == 0.0


def test_plain_parts_router_and_activation():
    y = torch.cat([torch.ones(1, 4, dtype=F64), 100.0 * torch.ones(1, 4, dtype=F64)], 1)
    assert torch.allclose(O.part_norm(y, 2, 0.0), torch.ones(1, 8, dtype=F64)) and not torch.allclose(O.part_norm(y, 1, 0.0), torch.ones(1, 8, dtype=F64))
    picks = O.route(torch.tensor([1.0, 3.0, 2.0, 3.0], dtype=F64), 2)
    assert [e for e, _ in picks] == [1, 3] and picks[0][1] == pytest.approx(0.5)
    assert float(O.gelu_tanh(torch.tensor(1.0, dtype=F64))) == pytest.approx(0.841192, abs=1e-6)


def test_plain_forward_is_causal_and_runs_every_branch():
    d = _cfg([PAR, SSM, dict(SSM, mlp=None), dict(PAR, mlp=dict(MOE, shared=None))])
    w = random_weights(TotatarConfig.from_dict(d), 1)
    toks = [3, 1, 4, 1, 5, 9, 2, 6]
    lay = []
    full = O.forward(d, w, toks, lay)
    assert full.shape == (8, 41) and len(lay) == 4
    assert torch.allclose(O.forward(d, w, toks[:5]), full[:5], atol=1e-9)
