"""`bench.py --design totatar`: prefill and decode throughput of the Totatar design at sizes that resemble a real model's layers (random
weights), next to Legavik -- the framework's closest model: attention and a matrix-state recurrence side by side, routed experts, float32
residual -- at equal width / heads / head and expert sizes, both through the same scheduler; plus the design's kernels one by one against
their roofline, with the like kernels of Legavik and, where Legavik has none, of Repepel (linear attention with fixed decays, shared
expert), Kinanex (selective scan, convolution) and Mutusun (two norms around the residual sum). Prints one JSON line. The default workload
of bench.py is untouched by this option.
"""
from __future__ import annotations

import math

from . import bench_kinanex, bench_legavik, bench_repepel, bench_seq
from .bench_seq import SIZES, VOCAB, _throughput, _time_us

# the sizes of `bench_legavik.LEGAVIK_SIZES` (width, heads x 128, key/value heads, window, experts) with a dense feed-forward size, a shared
# expert as large as a routed one, and a Mamba-2 mixer of twice the width: heads of 64, a state of 128, eight groups
TOTATAR_SIZES = {
    n: dict({k: v for k, v in s.items() if k not in ("rank", "groups", "keep_first", "latent", "side")}, ff=SIZES[n]["ff"], shared=s["moe"][1],
            ssm=(2 * s["width"] // 64, 8, 128, 64)) for n, s in bench_legavik.LEGAVIK_SIZES.items()
}


def totatar_config(s):
    """Four layers: parallel and Mamba-2 mixers in turn, a dense feed-forward first, routed experts after."""
    H, G, D = s["heads"], s["kv"], s["dim"]
    E, F, top = s["moe"]
    mh, mg, N, P = s["ssm"]
    moe = {"kind": "moe", "expert": {"ff": F}, "router": {"experts": E, "top": top}, "shared": {"ff": s["shared"]}}
    par = {"left": {"heads": H, "kv_heads": G, "dim": D, "vdim": D, "scale": D ** -0.5, "mask": {"size": s["window"]},
                    "rot": {"base": 500000.0, "dims": D, "scaling": {"factor": 4.0}}},
           "right": {"heads": H, "dim": D, "vdim": D, "decay": [math.exp(-1.0 / (4.0 * (i + 1))) for i in range(H)]},
           "left_scale": 0.8, "right_scale": 1.2}
    ssm = {"heads": mh, "groups": mg, "state": N, "vdim": P, "conv": s["conv"], "norm_groups": mg}
    layers = [{"type": "parallel", "mixer": par, "mlp": {"kind": "dense", "ff": s["ff"]}}, {"type": "mamba2", "mixer": ssm, "mlp": moe},
              {"type": "parallel", "mixer": par, "mlp": moe}, {"type": "mamba2", "mixer": ssm, "mlp": moe}]
    return {"architecture": "Totatar", "vocab": VOCAB, "width": s["width"], "norm": {"eps": 1e-5}, "layers": layers}


def _kernel_table(torch, s, hbm_gbs, bf16_tflops):
    """Each Totatar kernel at a prompt shape (2 048 tokens of one sequence) and a decode shape (64 sequences x 1 token with `window` +
    300 tokens behind it). Bytes: what the step must read and write once (projection rows, outputs, states), whatever the kernels keep in
    scratch. frac = achieved / measured peak of the binding resource."""
    from . import ops
    from .state import SequenceTable
    dev = "cuda"
    W, H, G, D, win, FF, FS, taps = (s[k] for k in ("width", "heads", "kv", "dim", "window", "ff", "shared", "conv"))
    E, F, top = s["moe"]
    mh, mg, N, P = s["ssm"]
    ctx, inner = win + 300, mh * P
    bf = torch.bfloat16
    rows = []

    def add(name, shape, us, nbytes=None, flops=None, note=None):
        e = {"kernel": name, "shape": shape, "us": round(us, 2)}
        if nbytes is not None:
            e["GBps"] = round(nbytes / us / 1e3, 1); e["frac_hbm"] = round(nbytes / us / 1e3 / hbm_gbs, 3)
        if flops is not None:
            e["TFLOPs"] = round(flops / us / 1e6, 1); e["frac_bf16"] = round(flops / us / 1e6 / bf16_tflops, 3)
        if note:
            e["note"] = note
        rows.append(e)

    nslots, cap = 64, 4096
    shapes = {"prompt": [(0, 2048)], "decode": [(ctx - 1 + 3 * k, 1) for k in range(64)]}
    ck = [(torch.randn(nslots, cap, G, D, device=dev) * 0.5).to(bf) for _ in range(2)]
    cv = [(torch.randn(nslots, cap, G, D, device=dev) * 0.5).to(bf) for _ in range(2)]
    fr = (500000.0 ** (-2.0 * torch.arange(D // 2, dtype=torch.float64) / D) / 4.0).float().to(dev)
    for label, segs in shapes.items():
        table = SequenceTable(nslots, dev, 2048)
        for k, (p0, _) in enumerate(segs):
            table.pos[table.open(k)] = p0
        meta = table.plan([(k, n) for k, (_, n) in enumerate(segs)])
        tab, T, nseg = meta.table, meta.ntok, len(segs)
        decode = label == "decode"
        positions = [p for p0, n in segs for p in range(p0, p0 + n)]
        nbuf = max(2, min(8, int(200e6 / (T * W * 12)) + 1))
        x = [torch.randn(T, W, device=dev) for _ in range(nbuf)]
        y = [torch.randn(T, W, device=dev).to(bf) for _ in range(nbuf)]
        h = [torch.empty(T, W, device=dev, dtype=bf) for _ in range(nbuf)]
        wv = torch.zeros(W, device=dev)
        us = _time_us(torch, [lambda i=i: ops.seq_sandwich_norm(x[i], 1e-5, y=y[i], post_w=wv, pre_w=wv, x_out=x[i], out=h[i]) for i in range(nbuf)])
        add("seq_sandwich_norm (norm of the result + residual + next input norm + cast)", f"{label} T={T} W={W}", us, nbytes=T * W * 12)
        pair = [torch.randn(T, top, W, device=dev).to(bf) for _ in range(max(2, nbuf // 2))]
        rw = torch.rand(T, top, device=dev)
        us = _time_us(torch, [lambda i=i: ops.seq_sandwich_norm(x[i], 1e-5, y=pair[i], y_w=rw, y2=y[i], post_w=wv, pre_w=wv, x_out=x[i], out=h[i])
                              for i in range(len(pair))])
        add("seq_sandwich_norm (weighted experts + shared expert)", f"{label} T={T} top={top}", us, nbytes=T * W * (12 + 2 * top))
        # left half
        ld = (H + 2 * G) * D
        pl = [torch.randn(T, ld, device=dev).to(bf) for _ in range(nbuf)]
        qf = [torch.empty(T, H, D, device=dev) for _ in range(2)]
        us = _time_us(torch, [lambda i=i: ops.seq_head_prep(pl[i], 0, H * D, (H + G) * D, qf[i % 2], ck[i % 2], cv[i % 2], tab, H, 1e-5, norm=False,
                                                            inv_freq=fr, rot_dims=D, pairing="interleaved") for i in range(nbuf)])
        add("seq_head_prep (interleaved rotary, no norm, cache rows)", f"{label} T={T}", us, nbytes=T * (ld * 2 + H * D * 4 + 2 * G * D * 2))
        qs = [torch.randn(T, H, D, device=dev) * 0.3 for _ in range(2)]
        out = torch.empty(T, H, D, device=dev, dtype=bf)
        sink = torch.zeros(H, device=dev)

        def attend(i):
            if decode:
                ops.seq_window_attention_mma(qs[i], ck[i], None, cv[i], out, tab, win, D ** -0.5, False, sink=sink)
            else:
                ops.seq_prompt_attention_mma(qs[i], ck[i], None, cv[i], out, 0, 0, win, D ** -0.5, sink=sink)

        us = _time_us(torch, [lambda i=i: attend(i) for i in range(2)])
        visible = sum(min(p + 1, win) for p in positions)
        if decode:
            add("seq_window_attention_mma, window + sink (heads of a group per CTA)", f"64 seqs x 1, {visible // T} keys each", us,
                nbytes=visible * G * 2 * D * 2)
        else:
            add("seq_prompt_attention_mma, window + sink (64 or 128 tokens per CTA)", f"T={T} window={win} H={H} G={G} D={D}", us,
                flops=4.0 * visible * H * D)
        # right half
        ldr = 4 * H * D
        pr = [torch.randn(T, ldr, device=dev).to(bf) for _ in range(nbuf)]
        dec = torch.full((H,), 0.98, device=dev)
        ldec = torch.log(dec)
        state = torch.zeros(nslots, H, D, D, device=dev)
        rec = torch.empty(T, H * D, device=dev)
        od = torch.empty(T, H * D, device=dev, dtype=bf)
        nw = torch.ones(H * D, device=dev)
        scratch = torch.empty(max(ops.seq_scalar_decay_scratch_bytes(T // 32, H, D, D), ops.seq_scalar_decay_scratch_bytes(T // 32, mh, N, P), 16),
                              dtype=torch.uint8, device=dev)

        def linear(i):
            ops.seq_scalar_decay(pr[i], 0, H * D, 2 * H * D, H, state, rec, meta, decay=dec, log_decay=ldec, scratch=scratch)
            ops.seq_part_norm(rec, nw, pr[i][:, 3 * H * D:], "sigmoid_after", od, 1e-5)

        us = _time_us(torch, [lambda i=i: linear(i) for i in range(nbuf)])
        add("seq_scalar_decay, fixed decays + seq_part_norm (silu, recurrence, norm over the heads, gate: " + ("2 launches)" if decode else "4 launches)"),
            f"{label} T={T} H={H} D={D}", us, nbytes=T * (ldr * 2 + H * D * 2) + (2 * nseg * H * D * D * 4 if decode else 0),
            flops=4.0 * T * H * D * D)
        # Mamba-2
        C = inner + 2 * mg * N
        ldm = inner + C + -(-mh // 8) * 8
        pm = [torch.randn(T, ldm, device=dev).to(bf) for _ in range(nbuf)]
        cw, cb = torch.randn(C, taps, device=dev) * 0.5, torch.zeros(C, device=dev)
        tail = torch.zeros(2, nslots, taps - 1, C, device=dev)
        hv = lambda v: torch.full((mh,), v, device=dev)
        dtb, al, dsk = hv(-2.5), hv(1.0), hv(1.0)
        mstate = torch.zeros(nslots, mh, N, P, device=dev)
        mrec = torch.empty(T, inner, device=dev)
        mo = torch.empty(T, inner, device=dev, dtype=bf)
        mn = torch.ones(inner, device=dev)
        co = torch.empty(T, C, device=dev, dtype=bf)
        if not decode:
            us = _time_us(torch, [lambda i=i: ops.seq_conv_act(pm[i][:, inner:inner + C], cw, cb, tail, co, tab) for i in range(nbuf)])
            add("seq_conv_act (convolution + bias + silu, a part of the next row)", f"{label} T={T} C={C} taps={taps}", us, nbytes=T * C * 4)
            us = _time_us(torch, [lambda i=i: ops.seq_part_norm(mrec, mn, pm[i][:, :inner], "silu_before", mo, 1e-5, parts=mg) for i in range(nbuf)])
            add("seq_part_norm (silu gate, norm in parts, a part of the next row)", f"{label} T={T} N={inner} parts={mg}", us, nbytes=T * inner * 8)

        def mamba(i):
            ops.seq_scalar_decay(pm[i], inner + inner + mg * N, inner + inner, inner, mg, mstate, mrec, meta, dt=pm[i][:, inner + C:inner + C + mh],
                                 dt_bias=dtb, A_log=al, D_skip=dsk, conv=(cw, cb, inner, tail), conv_out=co, scratch=scratch)
            ops.seq_part_norm(mrec, mn, pm[i][:, :inner], "silu_before", mo, 1e-5, parts=mg)

        us = _time_us(torch, [lambda i=i: mamba(i) for i in range(nbuf)])
        add("Mamba-2: seq_conv_act, seq_scalar_decay, seq_part_norm (" + ("2 launches)" if decode else "5 launches)"),
            f"{label} T={T} heads={mh} state={N} x {P} groups={mg}", us,
            nbytes=T * (ldm * 2 + inner * 2) + (2 * nseg * (mh * N * P + (taps - 1) * C) * 4 if decode else 0), flops=4.0 * T * mh * N * P)
        # feed-forward
        for hidden, act, what in ((FF, "gelu_tanh", "dense"), (FS, "silu", "shared expert")):
            gu = [torch.randn(T, 2 * hidden, device=dev).to(bf) for _ in range(2)]
            fo = torch.empty(T, hidden, device=dev, dtype=bf)
            us = _time_us(torch, [lambda i=i: ops.seq_glu(gu[i], fo, act) for i in range(2)])
            add(f"seq_glu ({act}, {what})", f"{label} T={T} F={hidden}", us, nbytes=T * hidden * 6)
        hh = torch.randn(T, W, device=dev).to(bf)
        rt, rb = torch.randn(E, W, device=dev) * 0.02, torch.zeros(E, device=dev)
        idx = torch.empty(T, top, dtype=torch.int32, device=dev)
        us = _time_us(torch, [lambda: ops.moe_route_chosen(hh, rt, idx, rw, bias=rb)] * 2)
        add("moe_route_chosen (bias, softmax over the chosen)", f"{label} T={T} R={E}", us, nbytes=T * W * 2 + E * W * 4)
        gu = [(torch.randn(E, 2 * F, W, device=dev) * 0.02).to(bf) for _ in range(2)]
        dn = [(torch.randn(E, W, F, device=dev) * 0.02).to(bf) for _ in range(2)]
        po = torch.empty(T, top, W, device=dev, dtype=bf)
        us = _time_us(torch, [lambda i=i: ops.moe_expert_grouped(hh, gu[i], dn[i], idx, po, E, F, 0.0, act="silu") for i in range(2)])
        if decode:
            touched = int(torch.unique(idx).numel())
            add("moe_expert_grouped, silu gate (sort + 2 tile GEMMs)", f"T={T} top={top}, {touched} of {E} experts touched", us,
                nbytes=touched * 3 * F * W * 2)
        else:
            add("moe_expert_grouped, silu gate (sort + 2 tile GEMMs)", f"T={T} top={top} E={E} F={F}", us, flops=6.0 * T * top * F * W)
        del x, y, h, pair, pl, pr, pm, gu, dn, scratch
    return rows


def run_totatar(args, peaks, clock_sampler_cls) -> dict:
    import torch
    from . import ops
    from .build import build_seq_library
    from .legavik import LegavikConfig, LegavikModel, random_weights as legavik_weights
    from .scheduler import Scheduler
    from .totatar import TotatarConfig, TotatarModel, random_weights
    build_seq_library()
    torch.cuda.set_device(0)
    hbm_gbs, bf16_tflops, peak_src = peaks
    bf16_tflops = bf16_tflops or 1590.0
    names = [n for n in (args.sizes.split(",") if args.sizes else TOTATAR_SIZES) if n in TOTATAR_SIZES]
    steps, warmup = args.steps, max(3, args.warmup)
    out = {}
    sampler = clock_sampler_cls(0)
    sampler.start()
    l0 = ops.seq_launch_count()
    for name in names:
        s = TOTATAR_SIZES[name]
        ctx = s["window"] + 300
        res = {"layers": 4, "sizes": {k: v for k, v in s.items()}}
        cfg = TotatarConfig.from_dict(totatar_config(s))
        model = TotatarModel(cfg, random_weights(cfg, 0), dtype=torch.bfloat16, device="cuda", n_slots=65, max_step_tokens=2048)
        res["totatar"] = {p: _throughput(torch, Scheduler(model, prefill_portion=p), VOCAB, 64, ctx, 4096, p, steps, warmup) for p in (2048, 256)}
        res["totatar"]["state_bytes_per_sequence"] = model.state_bytes_per_slot()
        del model
        torch.cuda.empty_cache()
        ls = bench_legavik.LEGAVIK_SIZES[name]
        lcfg = LegavikConfig.from_dict(bench_legavik.legavik_config(ls)).with_ranks(decay_rank=ls["rank"], gate_rank=ls["rank"])
        leg = LegavikModel(lcfg, legavik_weights(lcfg, 0), dtype=torch.bfloat16, device="cuda", n_slots=65, max_step_tokens=2048,
                           max_seq_tokens=4096 + 512)
        res["legavik"] = {p: _throughput(torch, Scheduler(leg, prefill_portion=p), VOCAB, 64, ctx, 4096, p, steps, warmup) for p in (2048, 256)}
        res["legavik"]["state_bytes_per_sequence"] = leg.state_bytes_per_slot()
        del leg
        torch.cuda.empty_cache()
        res["kernels"] = _kernel_table(torch, s, hbm_gbs, bf16_tflops)
        res["like_kernels_legavik"] = bench_legavik._kernel_table(torch, ls, hbm_gbs, bf16_tflops)
        for label, mod, sizes, keep in (("repepel", bench_repepel, bench_repepel.REPEPEL_SIZES, ("seq_lightning", "seq_silu_mul", "seq_act")),
                                        ("kinanex", bench_kinanex, bench_kinanex.KINANEX_SIZES, ("seq_conv_act", "seq_selective_scan")),
                                        ("mutusun", bench_seq, SIZES, ("seq_norm_conv",))):
            res["like_kernels_" + label] = [r for r in mod._kernel_table(torch, sizes[name], hbm_gbs, bf16_tflops) if r["kernel"].startswith(keep)]
            torch.cuda.empty_cache()
        out[name] = res
    clocks = sampler.stop()
    head = out[names[-1]]["totatar"][2048]
    return {"metric": "totatar_prefill_decode_tokens_per_s", "value": head["decode_tokens_per_s"], "unit": "tokens/s (decode, 64 sequences)",
            "n_gpus": 1, "steps": steps, "warmup": warmup, "ms_per_step": head["decode_ms_per_step"], "higher_is_better": True,
            "scaling": "weak", "vs_baseline": None, "dtype": "bf16 (float32 residual, norms, scores, weights, recurrences)", "data": "synthetic",
            "config": {"design": "totatar", "sizes": names, "weights": "random", "layers": 4,
                       "l2": "kernel timings rotate buffers larger than the L2 where the kernel streams from HBM"},
            "peaks": {"hbm_gbs": hbm_gbs, "bf16_tflops": bf16_tflops, "source": peak_src},
            "gpu_launches": ops.seq_launch_count() - l0, "clocks": clocks, "results": out}
