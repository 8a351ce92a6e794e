"""Host-side logic of the Legavik design (no GPU): configuration parsing and tensor names, registry entry, the number formats the
replay program accepts, the block tables of a step, and properties of the plain implementation that the GPU tests lean on."""
import json
import math

import pytest
import torch

from oracle import legavik_oracle as O
from qspec_b200 import registry
from qspec_b200.legavik import LegavikConfig, random_weights, rotary_amplitude, rotary_frequencies
from qspec_b200.state import SCAN_BLOCK, SCAN_SHORT, SequenceTable

F64 = torch.float64

MOE = {"kind": "moe", "expert": {"ff": 10}, "router": {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 2}}}
ATT = {"type": "attention", "mlp": MOE,
       "mixer": {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 6, "scale": 0.4, "mask": {"size": 5, "keep_first": 2},
                 "rot": {"base": 100.0, "dims": 4, "scaling": {"factor": 2.0, "original": 64, "fast": 4.0, "slow": 1.0}}}}
PAR = {"type": "parallel", "mlp": None,
       "mixer": {"left": {"heads": 4, "kv_heads": 2, "dim": 5, "vdim": 3, "conv": 2, "scale": 0.3, "q_temp": {"coef": 0.2, "every": 3}},
                 "right": {"heads": 4, "kv_heads": 2, "dim": 7, "vdim": 9, "conv": 3}, "left_scale": 0.75, "right_scale": 1.5}}


def _cfg(layers, width=32, vocab=41, softcap=9.0):
    return {"architecture": "Legavik", "vocab": vocab, "width": width, "norm": {"eps": 1e-5}, "logit_softcap": softcap, "layers": layers}


def test_configuration_round_trip_and_tensor_names():
    d = _cfg([ATT, PAR, dict(ATT, mlp=None), dict(PAR, mlp=MOE)])
    cfg = LegavikConfig.from_dict(d)
    assert LegavikConfig.from_dict(cfg.to_dict()) == cfg
    s = cfg.with_ranks(decay_rank=4, gate_rank=6).tensor_shapes()
    assert s["embed"] == (41, 32) and s["head"] == (41, 32) and s["final.norm"] == (32,) and s["final.norm.alpha"] == () and s["l0.norm1.b"] == (32,)
    assert s["l0.mix.q"] == (24, 32) and s["l0.mix.k"] == (12, 32) and "l0.mix.v" not in s and s["l0.mix.g"] == (4, 32) and s["l0.mix.o"] == (32, 24)
    assert s["l0.mlp.router"] == (6, 32) and s["l0.mlp.e5.gate"] == (10, 32) and s["l0.mlp.e0.down"] == (32, 10) and "l0.mlp.e6.up" not in s
    L, R = "l1.mix.left.", "l1.mix.right."
    assert s[L + "q"] == (20, 32) and s[L + "k.b"] == (10,) and s[L + "v.conv"] == (6, 2) and s[L + "q.norm"] == (5,) and s[L + "o"] == (32, 12)
    assert s[L + "o.b"] == (32,) and s[L + "g"] == (4, 32)
    assert s[R + "q"] == (14, 32) and s[R + "v.conv"] == (36, 3) and s[R + "b"] == (4, 32) and s[R + "A_log"] == (4,) and s[R + "norm"] == (9,)
    assert s[R + "a1"] == (4, 32) and s[R + "a2"] == (28, 4) and s[R + "dt_bias"] == (28,) and s[R + "g1"] == (6, 32) and s[R + "g2"] == (36, 6)
    assert s[R + "o"] == (32, 36) and "l1.norm2" not in s and "l2.mlp.router" not in s
    full = cfg.with_ranks(decay_rank=4, gate_rank=6)
    assert set(random_weights(full)) == set(s)
    assert cfg.with_ranks(random_weights(full)) == full                # the inner sizes come from a checkpoint's tensors
    with pytest.raises(ValueError):
        random_weights(cfg)
    # optional keys: no mask, no rotation, no temperature, no groups, no soft cap, key heads and sizes by default
    bare = {"type": "attention", "mixer": {"heads": 3, "dim": 4, "scale": 0.5},
            "mlp": {"kind": "moe", "expert": {"ff": 3}, "router": {"experts": 4, "top": 4}}}
    c2 = LegavikConfig.from_dict({k: v for k, v in _cfg([bare]).items() if k != "logit_softcap"})
    a, f = c2.layers[0].mixer.att, c2.layers[0].mlp
    assert (a.kv_heads, a.vdim, a.rot_dims, a.window, a.temp_every, c2.logit_softcap, f.groups, f.keep) == (3, 4, 0, None, 0, None, 1, 1)


@pytest.mark.parametrize("change", [
    lambda d: d["layers"][0].update(type="conv"),
    lambda d: d["layers"][0]["mixer"].update(kv_heads=3),
    lambda d: d["layers"][0]["mixer"].update(vdim=8),                   # the values are the keys
    lambda d: d["layers"][0]["mixer"]["rot"].update(dims=8),
    lambda d: d["layers"][0]["mlp"].update(kind="dense"),
    lambda d: d["layers"][0]["mlp"]["router"].update(top=5),            # more than the kept groups hold
    lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(count=4),
    lambda d: d["layers"][1]["mixer"]["right"].update(kv_heads=3),
    lambda d: d["layers"][1]["mixer"]["left"].update(conv=0),
])
def test_configuration_errors(change):
    d = json.loads(json.dumps(_cfg([ATT, PAR])))
    change(d)
    with pytest.raises(ValueError):
        LegavikConfig.from_dict(d)


def test_registry_and_number_formats(tmp_path):
    assert "Legavik" in registry.architectures()
    assert registry.supports_dtype("Legavik", "bfloat16") and registry.supports_dtype("Legavik", "float32")
    assert not registry.supports_dtype("Legavik", "float16")
    with open(tmp_path / "config.json", "w") as f:
        json.dump(_cfg([PAR]), f)
    from qspec_b200.trace import main
    assert main(["--model", str(tmp_path), "--dtype", "float16", "--out", str(tmp_path / "o")]) == 3


def test_stretched_frequencies_and_amplitude():
    """Fast pairs keep their frequency, slow ones are divided, a ramp between; both implementations agree; degenerate ramps."""
    for dims, base, sc in ((16, 1000.0, {"factor": 8.0, "original": 256, "fast": 8.0, "slow": 1.0}),
                           (12, 50.0, {"factor": 4.0, "original": 32, "fast": 32.0, "slow": 1.0}),       # lo would be negative
                           (8, 10.0, {"factor": 3.0, "original": 1e6, "fast": 32.0, "slow": 1.0}),        # hi would pass the last pair
                           (4, 1e5, {"factor": 2.0, "original": 7, "fast": 1.01, "slow": 1.0}), (10, 77.0, None)):
        got = rotary_frequencies(dims, base, sc)
        assert torch.allclose(got, torch.tensor(O.yarn_frequencies(dims, base, sc), dtype=F64), rtol=1e-12)
        assert rotary_amplitude(sc) == pytest.approx(O.yarn_amplitude(sc))
    sc = {"factor": 8.0, "original": 256, "fast": 8.0, "slow": 1.0}
    ratio = (rotary_frequencies(16, 1000.0, sc) / rotary_frequencies(16, 1000.0)).tolist()
    assert ratio[0] == 1.0 and ratio[-1] == pytest.approx(1 / 8) and any(0.13 < r < 0.99 for r in ratio)
    assert rotary_amplitude(sc) == pytest.approx(1.0 + 0.1 * math.log(8.0)) and rotary_amplitude(None) == 1.0


def test_block_tables_of_a_step():
    """Segments longer than SCAN_SHORT tokens are cut into blocks of SCAN_BLOCK from their own first row; short ones have none."""
    t = SequenceTable(8, "cpu", 256)
    lens = [1, 33, SCAN_SHORT, SCAN_SHORT + 1, 16, 2, 17]
    meta = t.plan([(k, n) for k, n in enumerate(lens)])
    begin, rows, starts, first = 0, [], [], []
    for n in lens:
        if n > SCAN_SHORT:
            starts.append(begin)
            first.append(len(rows))
            rows += list(range(begin, begin + n, SCAN_BLOCK))
        begin += n
    assert meta.block_rows.tolist() == rows and meta.long_starts.tolist() == starts and meta.long_block0.tolist() == first
    assert len(rows) <= sum(lens) // SCAN_SHORT                          # what the model reserves scratch for
    meta = t.plan([("x", 3)])
    assert meta.block_rows.numel() == meta.long_starts.numel() == 0


def test_block_count_never_exceeds_the_reserved_scratch():
    for n in range(SCAN_SHORT + 1, 300):
        assert -(-n // SCAN_BLOCK) <= n // SCAN_SHORT


def test_plain_delta_rule_decays_every_key_channel_on_its_own():
    """beta = 1 and unit keys along the axes: a value written for axis d is read back after n steps times the product of that axis'
    decays, whatever the others did."""
    T, D, DV = 5, 3, 2
    g = torch.rand(T, 1, D, generator=torch.Generator().manual_seed(0), dtype=F64)
    k = torch.zeros(T, 1, D, dtype=F64)
    k[0, 0, 1] = 1.0
    k[1:, 0, 2] = 1.0
    v = torch.zeros(T, 1, DV, dtype=F64)
    v[0, 0] = torch.tensor([2.0, -1.0], dtype=F64)
    q = torch.zeros(T, 1, D, dtype=F64)
    q[:, 0, 1] = 1.0
    o = O.delta_rule(q, k, v, torch.ones(T, 1, dtype=F64), g)
    keep = 1.0
    for t in range(T):
        keep = keep * float(g[t, 0, 1]) if t else 1.0
        assert torch.allclose(o[t, 0], v[0, 0] * keep, atol=1e-14)
    # carrying the state over a cut equals the whole sequence
    gen = torch.Generator().manual_seed(1)
    q, k = torch.randn(6, 2, D, generator=gen, dtype=F64), torch.randn(6, 2, D, generator=gen, dtype=F64)
    v, beta, g = torch.randn(6, 2, DV, generator=gen, dtype=F64), torch.rand(6, 2, generator=gen, dtype=F64), torch.rand(6, 2, D, generator=gen, dtype=F64)
    S = torch.zeros(2, D, DV, dtype=F64)
    parts = torch.cat([O.delta_rule(q[a:b], k[a:b], v[a:b], beta[a:b], g[a:b], S) for a, b in ((0, 4), (4, 6))])
    assert torch.allclose(O.delta_rule(q, k, v, beta, g), parts, atol=1e-12)


def test_plain_router_keeps_to_the_best_groups_and_normalises():
    z = torch.tensor([3.0, 0.0, 2.9, 2.8, 1.0, 2.95], dtype=F64)
    picks = O.route(z, top=2, groups=3, keep=2)                          # groups {0,1}, {2,3}, {4,5}: the best two are the first and the last
    assert [e for e, _ in picks] == [0, 5] and sum(w for _, w in picks) == pytest.approx(1.0)
    assert picks[0][1] / picks[1][1] == pytest.approx(math.exp(0.05))
    assert [e for e, _ in O.route(z, top=3)] == [0, 5, 2]


def test_plain_temperature_steps_and_window_mask():
    t = O.temperature(torch.arange(9), 0.5, 3)
    assert t[:2].tolist() == [1.0, 1.0] and t[2].item() == pytest.approx(1 + 0.5 * math.log(2)) and t[8].item() == pytest.approx(1 + 0.5 * math.log(4))
    n = 9
    q = torch.zeros(n, 1, 2, dtype=F64)
    v = torch.eye(n, dtype=F64)[:, None, :]
    o = O.masked_attention(q, torch.zeros(n, 1, 2, dtype=F64), v, 1.0, size=3, keep_first=2)      # equal weights: the mask shows
    assert (o[8, 0] > 0).tolist() == [j in (0, 1, 6, 7, 8) for j in range(n)]
    assert (o[3, 0] > 0).tolist() == [j in (0, 1, 2, 3) for j in range(n)]


def test_plain_forward_is_causal_and_runs_every_branch():
    d = _cfg([PAR, ATT, dict(PAR, mlp=MOE), dict(ATT, mlp=None)])
    w = random_weights(LegavikConfig.from_dict(d).with_ranks(decay_rank=3, gate_rank=2), 1)
    toks = [3, 1, 4, 1, 5, 9, 2, 6]
    lay = []
    full = O.forward(d, w, toks, lay)
    assert full.shape == (8, 41) and len(lay) == 4 and float(full.abs().max()) < 9.0
    assert torch.allclose(O.forward(d, w, toks[:5]), full[:5], atol=1e-9)
