"""Prefill / decode throughput of the Balivik stack (several residual streams; differential attention, fixed-decay linear attention and a
per-channel gated delta rule; dense feed-forwards and experts chosen by token id) beside the closest stacks on the same engine at equal layer
sizes, random weights, plus a per-kernel table: every kernel the stack added or extended, timed alone (CUDA events, L2 flushed between
iterations) with its algorithmic bytes or FLOPs as a fraction of the measured copy bandwidth / bf16 GEMM rate, next to the like kernel of
another stack on the same shapes.  Run through ``bench.py --config balivik``.

No one stack has both halves, so there are two comparisons: ``mixers`` — two attention layers and two recurrent layers with two dense
feed-forwards beside two Zanivik blocks (attention and recurrent layer side by side) with feed-forwards of the same weight count — and
``experts`` — four layers with two dense and two routed feed-forwards beside four Tusipel layers with the same feed-forwards."""
from __future__ import annotations

import json
import os

import torch

from . import benchmark_conv_latent as conv_latent
from . import benchmark_pairs as pairs
from .benchmark_pairs import VOCAB, _time, build, zanivik_config

STREAMS, TAPS, RANK = 2, 4, 128


def mixers(s):
    """The three mixers at the head counts and sizes of the Zanivik benchmark; a differential head's two maps split its key channels."""
    att = dict(heads=s["heads"], kv_heads=s["kv_heads"], dim=s["dim"] // 2, vdim=s["dim"], scale=(s["dim"] // 2) ** -0.5, diff=0.3,
               rot=dict(base=1e6, dims=s["dim"] // 2))
    lin = dict(heads=s["d_heads"], dim=s["d_dim"], vdim=s["d_vdim"], decay=[1.0 - 2.0 ** -(2 + 6.0 * i / s["d_heads"]) for i in range(s["d_heads"])])
    dlt = dict(heads=s["d_heads"], kv_heads=s["d_qk"], dim=s["d_dim"], vdim=s["d_vdim"], conv=4, decay_rank=RANK, gate_rank=RANK)
    return att, lin, dlt


def balivik_config(s, feed_forwards):
    att, lin, dlt = mixers(s)
    layers = [dict(type=t, mixer=m, mlp=f) for (t, m), f in zip((("attention", att), ("channel_delta", dlt), ("attention", att), ("lightning", lin)), feed_forwards)]
    return dict(architecture="Balivik", layers=layers, norm=dict(eps=1e-5), streams=STREAMS, canon=dict(taps=TAPS), logit_scale=1.0, vocab=VOCAB, width=s["width"])


def mixers_config(s):
    ff = dict(kind="dense", ff=s["ff"])
    return balivik_config(s, (ff, None, ff, None))


def experts_config(s, e):
    dense = dict(kind="dense", ff=e["dense_ff"])
    moe = dict(kind="moe", expert=dict(ff=e["ff"], limit=7.0), router=dict(experts=e["experts"], top=e["top"]))
    return balivik_config(s, (dense, moe, dense, moe))


def throughput(eng, batch, prompt, decode_steps, warmup):
    """tokens/s of one prefill step (batch rows x prompt tokens, host-resident ids in, tokens out) and of decode steps at that context."""
    ids = torch.randint(0, VOCAB, (batch, prompt), generator=torch.Generator().manual_seed(0))

    def prefill():
        for b in range(batch):
            eng.release(b)
        return eng.step([(b, ids[b].tolist(), ()) for b in range(batch)], sample=True)
    ms = _time(prefill, n=3, warm=max(1, min(warmup, 2)))
    tok = prefill()

    def decode(n):
        nonlocal tok
        for _ in range(n):
            tok = eng.step([(b, [tok[b]], ()) for b in range(batch)], sample=True)
    decode(warmup)
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    decode(decode_steps)
    e1.record()
    torch.cuda.synchronize()
    dms = e0.elapsed_time(e1)
    return dict(prefill_tok_s=batch * prompt * 1e3 / ms, decode_tok_s=batch * decode_steps * 1e3 / dms, decode_ms_per_step=dms / decode_steps)


def model_numbers(size, batch, prompt, decode_steps, warmup):
    s, e = pairs.SIZES[size], conv_latent.SIZES[size]
    room = prompt + decode_steps + warmup + 64
    out = {}
    for name, make in (("mixers_balivik", lambda: build(mixers_config(s), batch, room)), ("mixers_zanivik", lambda: build(zanivik_config(s), batch, room)),
                       ("experts_balivik", lambda: build(experts_config(s, e), batch, room)), ("experts_tusipel", lambda: conv_latent.build_tusipel(e, batch, room))):
        eng = make()
        for k, v in throughput(eng, batch, prompt, decode_steps, warmup).items():
            out[f"{name}_{k}"] = v
        del eng
        torch.cuda.empty_cache()
    return out


def kernel_table(size, batch, prompt, hbm_gbs, tflops):
    """Each kernel alone at the layers' shapes; after every new or extended kernel the like kernel of another stack on the same shapes.
    Prefill: batch x prompt tokens; decode: batch x 1 token at context ``prompt``."""
    from .. import ops
    s, ex = pairs.SIZES[size], conv_latent.SIZES[size]
    dev, bf = "cuda", torch.bfloat16
    flush = torch.empty(256 << 20, dtype=torch.uint8, device=dev)
    rows = []

    def run(name, fn, nbytes, flops=0.0, n=5):
        best = float("inf")
        for i in range(n + 2):
            flush.zero_()
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            fn()
            e1.record()
            torch.cuda.synchronize()
            if i >= 2:
                best = min(best, e0.elapsed_time(e1))
        rows.append(dict(kernel=name, ms=round(best, 4), gb=round(nbytes / 1e9, 4), frac_of_measured_hbm=round(nbytes / 1e6 / best / hbm_gbs, 3),
                         tflops=round(flops / 1e9 / best, 1), frac_of_measured_bf16=round(flops / 1e9 / best / tflops, 4)))

    W, H, G, D2, page = s["width"], s["heads"], s["kv_heads"], s["dim"], 64
    D = D2 // 2
    dh, dq, dD, dV = s["d_heads"], s["d_qk"], s["d_dim"], s["d_vdim"]
    nh, P, N, Gm = s["m_heads"], s["m_dim"], s["state"], s["groups"]
    E, k, F = ex["experts"], ex["top"], ex["ff"]
    rnd = lambda *shape, dt=bf: torch.randn(*shape, device=dev, dtype=dt)          # noqa: E731
    f32 = lambda *shape: torch.randn(*shape, device=dev)                           # noqa: E731
    for phase, T, ctx0 in (("prefill", prompt, 0), ("decode", 1, prompt)):
        B = batch
        R = B * T
        full = lambda v: torch.full((B,), v, dtype=torch.int32, device=dev)        # noqa: E731
        ctx, ql, lines = full(ctx0), full(T), torch.arange(B, dtype=torch.int32, device=dev)
        nblk = -(-(ctx0 + T) // page)
        table = torch.arange(B * nblk, dtype=torch.int32, device=dev).view(B, nblk)
        # residual streams
        for S in (STREAMS, 4):
            x, y = f32(B, T, S, W), rnd(B, T, W)
            mix, ow, iw, one, cw = f32(S, S), f32(S), f32(S), torch.ones(1, device=dev), f32(W, TAPS) * 0.1
            st = torch.zeros(B + 1, TAPS - 1, W, device=dev)
            nb = R * W * (4 * S * 2 + 2 + 2)
            run(f"{phase}: stream_mix_norm_conv ({S} streams, {TAPS} taps, carried rows advanced)",
                lambda: ops.stream_mix_norm_conv(x, y, mix, ow, iw, one, cw, st, lines, ctx, ql, 1e-5, bf), nb)
            run(f"{phase}: stream_mix_norm_conv ({S} streams, no convolution)",
                lambda: ops.stream_mix_norm_conv(x, y, mix, ow, iw, one, None, None, None, ctx, ql, 1e-5, bf), nb)
        x1, w = f32(B, T, W), torch.ones(W, device=dev)

        def tusipel_read():
            sn, _ = ops.stream_norm_conv(x1, (y,), w, cw, st, lines, ctx, ql, 1e-5, bf)
            ops.short_conv_update(sn, st, lines, ctx, ql)
        run(f"{phase}: stream_norm_conv + short_conv_update (Tusipel: one stream)", tusipel_read, R * W * (4 + 4 + 2 + 2))
        run(f"{phase}: stream_add_rmsnorm (Sodudra: one stream, no convolution)", lambda: ops.stream_add_rmsnorm(x1, (y,), weight=w, eps=1e-5, lp_dtype=bf),
            R * W * (4 + 4 + 2 + 2))
        # attention
        C = 2 * D * (H + G) + G * D2
        p = rnd(B, T, C)
        cos, sin = f32(B, T, D // 2), f32(B, T, D // 2)
        kc, vc = rnd(B * nblk, page, 2 * G, D), rnd(B * nblk, page, G, D2)
        run(f"{phase}: head_norm_rope_append (two maps of {D}, shared values)",
            lambda: ops.head_norm_rope_append(p, 2 * H, 2 * G, D, D2, cos, sin, None, None, 0, 1e-5, False, kc, vc, table, ctx, ql, n_v=G), R * C * 2 * 2)
        kz, vz = rnd(B * nblk, page, G, D2), rnd(B * nblk, page, G, D2)
        cz, sz = f32(B, T, D2 // 2), f32(B, T, D2 // 2)
        run(f"{phase}: head_norm_rope_append (Zanivik: norm after rotation, heads of {D2})",
            lambda: ops.head_norm_rope_append(p, H, G, D2, D2, cz, sz, None, None, 2, 1e-5, False, kz, vz, table, ctx, ql), R * C * 2 * 2)
        q = rnd(B, T, 2 * H, D)
        lam = torch.full((1,), 0.3, device=dev)
        visible = sum(t + 1 + ctx0 for t in range(T)) * B
        nb = B * (ctx0 + T) * G * (2 * D + D2) * 2 + R * H * (2 * D + D2) * 2
        run(f"{phase}: paged_diff_attention ({H}/{G} heads, two maps of {D}, values of {D2})",
            lambda: ops.paged_diff_attention(q, kc, vc, table, ctx, ql, D ** -0.5, lam, 0.7, 1e-5), nb, flops=4.0 * visible * H * (D + D2))
        qz = q.view(B, T, H, D2)
        run(f"{phase}: paged_window_attention (Zanivik without window: {H}/{G} heads of {D2})",
            lambda: ops.paged_window_attention(qz, kz, vz, table, ctx, ql, D2 ** -0.5, None, 0, 0), nb, flops=4.0 * visible * H * D2)
        # per-channel delta rule
        Cd = 2 * dq * dD + dh * dV
        pd, a = rnd(B, T, Cd + dh + 2 * RANK), rnd(B, T, dh * (dD + dV))
        cwd, cst = f32(Cd, 4) * 0.3, torch.zeros(B + 1, 3, Cd, device=dev, dtype=bf)
        Al, db = torch.zeros(dh, device=dev), torch.full((dh * dD,), -2.0, device=dev)
        run(f"{phase}: delta_front (convolutions, unit norms, {dh * dD} decays, carried rows advanced)",
            lambda: ops.delta_front(pd, pd[..., Cd:Cd + dh], a[..., :dh * dD], cwd, Al, db, cst, lines, ctx, ql, dh, dq, dD, dV), R * (Cd * 6 + dh * dD * 6))

        def zanivik_front():
            ops.short_conv(pd[..., :Cd], cwd, None, cst, lines, ctx, ql, True)
            ops.short_conv_update(pd[..., :Cd], cst, lines, ctx, ql)
        run(f"{phase}: short_conv + SiLU + short_conv_update (Zanivik)", zanivik_front, R * Cd * 6)
        qkv, g, be = f32(B, T, Cd) * 0.1, torch.rand(B, T, dh * dD, device=dev) * 0.1 + 0.9, torch.rand(B, T, dh, device=dev)
        S1, S2 = torch.zeros(B + 1, dh, dV, dD, device=dev), torch.zeros(B + 1, dh, dD, dV, device=dev)
        run(f"{phase}: channel_delta_scan ({dh} heads x {dD} x {dV})", lambda: ops.channel_delta_scan(qkv, g, be, S1, lines, ctx, ql, dh, dq, dD, dV),
            R * (Cd + dh * dD + dh * dV) * 4 + B * dh * dD * dV * 8, flops=7.0 * R * dh * dD * dV, n=3)
        Az = torch.full((dh,), -2.0, device=dev)
        run(f"{phase}: gated_delta_scan (Zanivik)",
            lambda: ops.gated_delta_scan(qkv, pd[..., Cd:Cd + dh], pd[..., Cd + dh:Cd + 2 * dh], Al, Az, S2, lines, ctx, ql, dh, dq, dD, dV),
            R * (Cd + dh * dV) * 4 + B * dh * dD * dV * 8, flops=6.0 * R * dh * dD * dV, n=3)
        od, nw, gate = f32(B, T, dh * dV), torch.ones(dV, device=dev), a[..., dh * dD:]
        run(f"{phase}: head_rmsnorm_gate (sigmoid; the same kernel in both stacks)", lambda: ops.head_rmsnorm_gate(od, nw, dh, 1e-5, gate, "sigmoid", bf), R * dh * dV * 8)
        # fixed decays
        inner = dh * dV
        pl = rnd(B, T, dh * (2 * dD + dV) + inner)
        dec = torch.linspace(0.7, 0.999, dh, device=dev)
        run(f"{phase}: decay_scan ({dh} heads x {dD} x {dV})", lambda: ops.decay_scan(pl, dec, S1, lines, ctx, ql, dh, dD, dV),
            R * (dh * (2 * dD + dV) * 2 + inner * 4) + B * dh * dD * dV * 8, flops=4.0 * R * dh * dD * dV, n=3)
        mi, Cm = nh * P, nh * P + 2 * Gm * N
        pm, xBC = rnd(B, T, mi + Cm + nh), f32(B, T, Cm) * 0.3
        Am, dm, Dk, Sm = torch.zeros(nh, device=dev), torch.full((nh,), -2.0, device=dev), torch.ones(nh, device=dev), torch.zeros(B + 1, nh, N, P, device=dev)
        run(f"{phase}: ssd_scan (Zanivik / Fetodra: {nh} heads x {N} x {P})",
            lambda: ops.ssd_scan(xBC, pm[..., mi + Cm:], pm[..., :mi], Am, dm, Dk, Sm, lines, ctx, ql, nh, P, N, Gm),
            R * (Cm * 4 + mi * 6) + B * nh * N * P * 8, flops=4.0 * R * nh * N * P, n=3)
        yv, wg, gl = f32(B, T, inner), torch.ones(inner, device=dev), pl[..., dh * (2 * dD + dV):]
        run(f"{phase}: group_rmsnorm with a gate", lambda: ops.group_rmsnorm(yv, wg, 1, 1e-5, bf, gl, "sigmoid"), R * inner * 8)
        run(f"{phase}: group_rmsnorm (Zanivik / Fetodra)", lambda: ops.group_rmsnorm(yv, wg, 1, 1e-5, bf), R * inner * 6)
        # experts
        xm, gu, dn = rnd(R, W), rnd(E, 2 * F, W) * 0.02, rnd(E, W, F) * 0.02
        tab = ((torch.arange(VOCAB, device=dev).view(-1, 1) * k + torch.arange(k, device=dev)) % E).int()
        ids = torch.randint(0, VOCAB, (B, T), device=dev, dtype=torch.int32)
        run(f"{phase}: table_route", lambda: ops.table_route(tab, ids, ql), R * (4 + k * 12))
        rw = f32(E, W)
        run(f"{phase}: router_topk (Tusipel: scores)", lambda: ops.router_topk(xm, rw, k, "softmax", False), R * W * 2, flops=2.0 * R * W * E)
        tw, ti = ops.table_route(tab, ids, ql)
        used = min(E, R * k)
        nb, fl = (used * 3 * F * W + R * W * 2) * 2, 6.0 * R * k * F * W
        run(f"{phase}: experts, clamped gate product", lambda: ops.moe_experts(xm, gu, dn, tw, ti, "clamped_glu", act_params=(7.0, 1.702)), nb, flops=fl)
        run(f"{phase}: experts, SiLU (Tusipel)", lambda: ops.moe_experts(xm, gu, dn, tw, ti, "silu_mul"), nb, flops=fl)
    return rows


def run(size="small", batch=4, prompt=1024, decode_steps=32, warmup=3):
    peaks = {}
    p = os.path.join(os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__)))), "MEASURED_PEAKS.json")
    if os.path.isfile(p):
        with open(p) as f:
            peaks = json.load(f)
    hbm, tf = float(peaks.get("hbm_gbs", 6650.0)), float(peaks.get("bf16_tflops", 1590.0))
    res = dict(size=size, shapes=dict(pairs.SIZES[size], streams=STREAMS, taps=TAPS, rank=RANK), expert_shapes=conv_latent.SIZES[size], batch=batch,
               prompt=prompt, decode_steps=decode_steps, hbm_gbs=hbm, bf16_tflops=tf, peaks_source="measured" if peaks else "fallback")
    res.update(model_numbers(size, batch, prompt, decode_steps, warmup))
    res["kernels"] = kernel_table(size, batch, prompt, hbm, tf)
    return res
