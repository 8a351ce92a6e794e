"""`bench.py --design legavik`: prefill and decode throughput of the Legavik design at sizes that resemble a real model's layers (random
weights), next to Kinanex -- the framework's closest model: full-length attention over convolved or normed heads, a gated delta rule
with short convolutions, float32 residual -- at equal width / heads / head sizes, both through the same scheduler; plus the design's
kernels one by one against their roofline, with the like kernels of Kinanex and, for window attention and routed experts (which
Kinanex has not), of Pitudra from `bench_seq`. Prints one JSON line. The default workload of bench.py is untouched by this option.
"""
from __future__ import annotations

from .bench_kinanex import KINANEX_SIZES, _kernel_table as _kinanex_kernel_table, kinanex_config
from .bench_seq import PITUDRA_SIZES, VOCAB, _pitudra_kernel_table, _throughput, _time_us

# the sizes of `bench_seq.PITUDRA_SIZES` (width, heads x 128, key/value heads, window, experts); the delta half has the full number of
# value heads over half as many query / key heads, as the delta layers of `bench_kinanex`
LEGAVIK_SIZES = {
    "w2048": dict(PITUDRA_SIZES["w2048"], conv=4, rank=128, groups=(4, 2), keep_first=4),
    "w4096": dict(PITUDRA_SIZES["w4096"], conv=4, rank=128, groups=(4, 2), keep_first=4),
}


def legavik_config(s):
    """Four layers: window attention and parallel layers in turn, every one with routed experts except the third."""
    H, G, D = s["heads"], s["kv"], s["dim"]
    E, F, top = s["moe"]
    count, keep = s["groups"]
    moe = {"kind": "moe", "expert": {"ff": F}, "router": {"experts": E, "top": top, "groups": {"count": count, "keep": keep}}}
    att = {"heads": H, "kv_heads": G, "dim": D, "vdim": D, "scale": D ** -0.5, "mask": {"size": s["window"], "keep_first": s["keep_first"]},
           "rot": {"base": 500000.0, "dims": D, "scaling": {"factor": 8.0, "original": 8192, "fast": 32.0, "slow": 1.0}}}
    par = {"left": {"heads": H, "kv_heads": G, "dim": D, "vdim": D, "scale": D ** -0.5, "conv": s["conv"], "q_temp": {"coef": 0.1, "every": 1024}},
           "right": {"heads": H, "kv_heads": H // 2, "dim": D, "vdim": D, "conv": s["conv"]}, "left_scale": 0.8, "right_scale": 1.2}
    layers = [{"type": "attention", "mixer": att, "mlp": moe}, {"type": "parallel", "mixer": par, "mlp": moe},
              {"type": "attention", "mixer": att, "mlp": None}, {"type": "parallel", "mixer": par, "mlp": moe}]
    return {"architecture": "Legavik", "vocab": VOCAB, "width": s["width"], "norm": {"eps": 1e-5}, "logit_softcap": 30.0, "layers": layers}


def _kernel_table(torch, s, hbm_gbs, bf16_tflops):
    """Each Legavik kernel at a prompt shape (2 048 tokens of one sequence) and a decode shape (64 sequences x 1 token with `window` +
    300 rows behind it). frac = achieved / measured peak of the binding resource."""
    from . import ops
    from .state import SequenceTable
    dev = "cuda"
    W, H, G, D, win = s["width"], s["heads"], s["kv"], s["dim"], s["window"]
    ctx, taps, keep_first = win + 300, s["conv"], s["keep_first"]
    E, F, top = s["moe"]
    count, keep = s["groups"]
    GD = H // 2                                             # query / key heads of the delta half
    bf = torch.bfloat16
    full = 1 << 30
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
    fr = (500000.0 ** (-2.0 * torch.arange(D // 2, dtype=torch.float64) / D)).float().to(dev)
    for label, segs in shapes.items():
        table = SequenceTable(nslots, dev, 2048)
        for k, (p0, _) in enumerate(segs):
            table.pos[table.open(k)] = p0
        meta = table.plan([(k, n) for k, (_, n) in enumerate(segs)])
        tab, T, nseg = meta.table, meta.ntok, len(segs)
        positions = [p for p0, n in segs for p in range(p0, p0 + n)]
        nbuf = max(2, min(8, int(200e6 / (T * W * 12)) + 1))
        x = [torch.randn(T, W, device=dev) for _ in range(nbuf)]
        y = [torch.randn(T, W, device=dev).to(bf) for _ in range(nbuf)]
        h = [torch.empty(T, W, device=dev, dtype=bf) for _ in range(nbuf)]
        wv, bv = torch.ones(W, device=dev), torch.zeros(W, device=dev)
        us = _time_us(torch, [lambda i=i: ops.seq_residual_tanh(x[i], 0.5, wv, bv, y=y[i], y_bias=bv, x_out=x[i], out=h[i]) for i in range(nbuf)])
        add("seq_residual_tanh (residual + output bias + tanh norm + cast)", f"{label} T={T} W={W}", us, nbytes=T * W * 12)
        pair = [torch.randn(T, top, W, device=dev).to(bf) for _ in range(max(2, nbuf // 2))]
        rw = torch.rand(T, top, device=dev)
        us = _time_us(torch, [lambda i=i: ops.seq_residual_tanh(x[i], 0.5, wv, bv, y=pair[i], y_w=rw, x_out=x[i], out=h[i]) for i in range(len(pair))])
        add("seq_residual_tanh (weighted sum of the experts' parts)", f"{label} T={T} top={top}", us, nbytes=T * W * (10 + 2 * top))
        # window attention
        ld = (H + G) * D + H
        pp = [torch.randn(T, ld, device=dev).to(bf) for _ in range(nbuf)]
        qf = [torch.empty(T, H, D, device=dev) for _ in range(2)]
        us = _time_us(torch, [lambda i=i: ops.seq_head_prep(pp[i], 0, H * D, None, qf[i % 2], ck[i % 2], cv[i % 2], tab, H, 1e-5, norm_last=True,
                                                            inv_freq=fr, rot_dims=D, rot_amp=1.2, keep_first=keep_first) for i in range(nbuf)])
        add("seq_head_prep (rotary with amplitude + head norms + cache rows, values = keys)", f"{label} T={T}", us,
            nbytes=T * (ld * 2 + H * D * 4 + 2 * G * D * 2))
        qs = [torch.randn(T, H, D, device=dev) * 0.3 for _ in range(2)]
        out = torch.empty(T, H, D, device=dev, dtype=bf)
        gate = torch.randn(T, H, device=dev).to(bf)

        def attend(i, window, kf):
            kw = dict(gate=gate, gate_per_head=True, keep_first=kf)
            if label == "prompt":
                ops.seq_prompt_attention_mma(qs[i], ck[i], None, cv[i], out, 0, 0, window, D ** -0.5, **kw)
            else:
                ops.seq_window_attention_mma(qs[i], ck[i], None, cv[i], out, tab, window, D ** -0.5, False, **kw)

        for name, window, kf in (("window + kept tokens", win, keep_first), ("whole sequence", full, 0)):
            us = _time_us(torch, [lambda i=i: attend(i, window, kf) for i in range(2)])
            visible = sum(min(p + 1, window + min(kf, max(p + 1 - window, 0))) for p in positions)
            if label == "prompt":
                add(f"seq_prompt_attention_mma, {name}, gate per head (64 or 128 tokens per CTA)", f"T={T} window={min(window, T)} H={H} G={G} D={D}", us,
                    flops=4.0 * visible * H * D)
            else:
                add(f"seq_window_attention_mma, {name}, gate per head (heads of a group per CTA)", f"64 seqs x 1, {visible // T} keys each", us,
                    nbytes=visible * G * 2 * D * 2)
        # left half of a parallel layer
        CL = (H + 2 * G) * D
        pl = [torch.randn(T, CL, device=dev).to(bf) for _ in range(nbuf)]
        cw, tail = torch.randn(taps, CL, device=dev) * 0.5, torch.zeros(2, nslots, taps - 1, CL, device=dev)
        qn = torch.ones(D, device=dev)
        us = _time_us(torch, [lambda i=i: ops.seq_head_prep(pl[i], 0, H * D, (H + G) * D, qf[i % 2], ck[i % 2], cv[i % 2], tab, H, 1e-5, conv_w=cw,
                                                            tail=tail, qn_w=qn, kn_w=qn, temp_coef=0.1, temp_every=1024) for i in range(nbuf)])
        add("seq_head_prep (convolution + head norms + temperature + cache rows)", f"{label} T={T} C={CL} taps={taps}", us,
            nbytes=T * (CL * 2 + H * D * 4 + 2 * G * D * 2) + (nseg * 2 * (taps - 1) * CL * 4 if label == "decode" else 0))
        # right half
        CR = 2 * GD * D + H * D
        pr = [torch.randn(T, CR + H, device=dev).to(bf) for _ in range(nbuf)]
        cwr, tailr = torch.randn(taps, CR, device=dev) * 0.5, torch.zeros(2, nslots, taps - 1, CR, device=dev)
        dec = [torch.randn(T, H * D, device=dev) for _ in range(nbuf)]
        al, db = torch.zeros(H, device=dev), torch.zeros(H * D, device=dev)
        gt = torch.randn(T, H * D, device=dev).to(bf)
        state = torch.zeros(nslots, H, D, D, device=dev)
        od = torch.empty(T, H * D, device=dev, dtype=bf)
        scratch = torch.empty(max(ops.seq_delta_channel_scratch_bytes(T // 8, T, H, D, D), 16), dtype=torch.uint8, device=dev)
        us = _time_us(torch, [lambda i=i: ops.seq_delta_channel(pr[i], CR, cwr, tailr, dec[i], al, db, qn, gt, state, od, meta, GD, 1e-5,
                                                                scratch=scratch) for i in range(nbuf)])
        add("seq_delta_channel (convolution, unit vectors, gates, recurrence, head norm + gate: " + ("3 launches)" if label == "prompt" else "1 launch)"),
            f"{label} T={T} H={H} D={D}", us,
            nbytes=T * (CR * 2 + H * D * (4 + 2 + 2)) + (2 * nseg * (H * D * D + (taps - 1) * CR) * 4 if label == "decode" else 0),
            flops=6.0 * T * H * D * D, note="blocks of 16 tokens in sequence, H x DV/16 CTAs per sequence" if label == "prompt" else None)
        # experts
        hh = torch.randn(T, W, device=dev).to(bf)
        rt = torch.randn(E, W, device=dev) * 0.02
        idx = torch.empty(T, top, dtype=torch.int32, device=dev)
        us = _time_us(torch, [lambda: ops.moe_route_grouped(hh, rt, None, idx, rw, score="softmax", groups=count, keep=keep, group_top=1,
                                                            normalize=True)] * 2)
        add("moe_route_grouped (softmax, groups, normalised weights)", f"{label} T={T} R={E}", us, nbytes=T * W * 2 + E * W * 4)
        gu = [(torch.randn(E, 2 * F, W, device=dev) * 0.02).to(bf) for _ in range(2)]
        dn = [(torch.randn(E, W, F, device=dev) * 0.02).to(bf) for _ in range(2)]
        po = torch.empty(T, top, W, device=dev, dtype=bf)
        us = _time_us(torch, [lambda i=i: ops.moe_expert_grouped(hh, gu[i], dn[i], idx, po, E, F, 0.0, act="silu") for i in range(2)])
        if label == "prompt":
            add("moe_expert_grouped, silu gate (sort + 2 tile GEMMs)", f"T={T} top={top} E={E} F={F}", us, flops=6.0 * T * top * F * W)
        else:
            touched = int(torch.unique(idx).numel())
            add("moe_expert_grouped, silu gate (sort + 2 tile GEMMs)", f"T={T} top={top}, {touched} of {E} experts touched", us,
                nbytes=touched * 3 * F * W * 2)
        lg = torch.randn(T if label == "decode" else 64, VOCAB, device=dev)
        us = _time_us(torch, [lambda: ops.seq_softcap(lg, 30.0)] * 2)
        add("seq_softcap", f"{lg.shape[0]} rows of {VOCAB}", us, nbytes=lg.numel() * 8, note="fits the L2")
        del x, y, h, pair, pp, pl, pr, dec, gu, dn, scratch
    return rows


def run_legavik(args, peaks, clock_sampler_cls) -> dict:
    import torch
    from . import ops
    from .build import build_seq_library
    from .kinanex import KinanexConfig, KinanexModel, random_weights as kinanex_weights
    from .legavik import LegavikConfig, LegavikModel, random_weights
    from .scheduler import Scheduler
    build_seq_library()
    torch.cuda.set_device(0)
    hbm_gbs, bf16_tflops, peak_src = peaks
    bf16_tflops = bf16_tflops or 1590.0
    names = [n for n in (args.sizes.split(",") if args.sizes else LEGAVIK_SIZES) if n in LEGAVIK_SIZES]
    steps, warmup = args.steps, max(3, args.warmup)
    out = {}
    sampler = clock_sampler_cls(0)
    sampler.start()
    l0 = ops.seq_launch_count()
    for name in names:
        s = LEGAVIK_SIZES[name]
        ctx = s["window"] + 300
        res = {"layers": 4, "sizes": {k: v for k, v in s.items()}}
        cfg = LegavikConfig.from_dict(legavik_config(s)).with_ranks(decay_rank=s["rank"], gate_rank=s["rank"])
        model = LegavikModel(cfg, random_weights(cfg, 0), dtype=torch.bfloat16, device="cuda", n_slots=65, max_step_tokens=2048,
                             max_seq_tokens=4096 + 512)
        res["legavik"] = {p: _throughput(torch, Scheduler(model, prefill_portion=p), VOCAB, 64, ctx, 4096, p, steps, warmup) for p in (2048, 256)}
        res["legavik"]["state_bytes_per_sequence"] = model.state_bytes_per_slot()
        del model
        torch.cuda.empty_cache()
        kcfg = KinanexConfig.from_dict(kinanex_config(KINANEX_SIZES[name]))
        kin = KinanexModel(kcfg, kinanex_weights(kcfg, 0), dtype=torch.bfloat16, device="cuda", n_slots=65, max_step_tokens=2048,
                           max_seq_tokens=4096 + 512)
        res["kinanex"] = {p: _throughput(torch, Scheduler(kin, prefill_portion=p), VOCAB, 64, ctx, 4096, p, steps, warmup) for p in (2048, 256)}
        res["kinanex"]["state_bytes_per_sequence"] = kin.state_bytes_per_slot()
        del kin
        torch.cuda.empty_cache()
        res["kernels"] = _kernel_table(torch, s, hbm_gbs, bf16_tflops)
        res["like_kernels_kinanex"] = _kinanex_kernel_table(torch, KINANEX_SIZES[name], hbm_gbs, bf16_tflops)
        res["like_kernels_pitudra"] = _pitudra_kernel_table(torch, PITUDRA_SIZES[name], hbm_gbs, bf16_tflops)
        out[name] = res
    clocks = sampler.stop()
    head = out[names[-1]]["legavik"][2048]
    return {"metric": "legavik_prefill_decode_tokens_per_s", "value": head["decode_tokens_per_s"], "unit": "tokens/s (decode, 64 sequences)",
            "n_gpus": 1, "steps": steps, "warmup": warmup, "ms_per_step": head["decode_ms_per_step"], "higher_is_better": True,
            "scaling": "weak", "vs_baseline": None, "dtype": "bf16 (float32 residual, norms, scores, weights, recurrences)", "data": "synthetic",
            "config": {"design": "legavik", "sizes": names, "weights": "random", "layers": 4,
                       "l2": "kernel timings rotate buffers larger than the L2 where the kernel streams from HBM"},
            "peaks": {"hbm_gbs": hbm_gbs, "bf16_tflops": bf16_tflops, "source": peak_src},
            "gpu_launches": ops.seq_launch_count() - l0, "clocks": clocks, "results": out}
