"""Prefill / decode throughput of the Navulorn stack (post-norm blocks over window attention, latent attention and matrix memories; dense and
routed feed-forwards; bigram embeddings) beside the closest stacks on the same engine at equal layer sizes, random weights, plus a per-kernel
table: every kernel the stack added or extended, timed alone (CUDA events, L2 flushed between iterations) with its algorithmic bytes or FLOPs
as a fraction of the measured copy bandwidth / bf16 GEMM rate, next to the like kernel of another stack on the same shapes.  Run through
``bench.py --config navulorn``.

No one stack has every kind of layer, so there are two comparisons: ``memory`` — two attention layers with dense feed-forwards and two matrix
memories beside the mixers of the Balivik benchmark (attention, per-channel delta rule, attention, fixed decays; same head sizes and
feed-forwards, no attention window) — and ``latent`` — two latent and two grouped-query attention layers with two dense and two routed
feed-forwards beside four Tusipel layers of the same kinds."""
from __future__ import annotations

import json
import os

import torch

from . import benchmark_conv_latent as conv_latent
from . import benchmark_pairs as pairs
from .benchmark_pairs import VOCAB, build
from .benchmark_streams import mixers_config as balivik_mixers
from .benchmark_streams import throughput

BIGRAM = dict(buckets=65521, mul_prev=37, mul_cur=11)
LLAMA31 = dict(factor=8.0, low=1.0, high=4.0, original=8192)
GATE_CAP = 15.0


def config(width, layers):
    return dict(architecture="Navulorn", layers=layers, norm=dict(eps=1e-6), postln_alpha=1.5, logit_softcap=30.0, vocab=VOCAB, width=width,
                embedding=dict(scale=1.0, bigram=BIGRAM))


def attention(s, window):
    return dict(heads=s["heads"], kv_heads=s["kv_heads"], dim=s["dim"], vdim=s.get("vdim", s["dim"]), scale=s["dim"] ** -0.5, mask=dict(size=window),
                rot=dict(base=5e5, dims=s["dim"], scaling=LLAMA31))


def memory_config(s):
    mem = dict(heads=s["d_heads"], dim=s["d_dim"], vdim=s["d_vdim"], gate_cap=GATE_CAP)
    ff = dict(kind="dense", ff=s["ff"])
    return config(s["width"], [dict(type="attention", mixer=attention(s, 1 << 20), mlp=ff), dict(type="mlstm", mixer=mem, mlp=None)] * 2)


def latent_config(e):
    lat = dict(heads=e["heads"], dim=e["dim"], rot_dim=e["rot"], vdim=e["vdim"], kv_rank=e["rank"], scale=(e["dim"] + e["rot"]) ** -0.5,
               mask=dict(size=e["window"]), rot=dict(base=10000.0, dims=e["rot"]))
    dense = dict(kind="dense", ff=e["dense_ff"])
    moe = dict(kind="moe", expert=dict(ff=e["ff"]), router=dict(experts=e["experts"], top=e["top"]))
    att = attention(e, e["chunk"])
    return config(e["width"], [dict(type="latent_attention", mixer=lat, mlp=dense), dict(type="attention", mixer=att, mlp=moe),
                               dict(type="attention", mixer=att, mlp=dense), dict(type="latent_attention", mixer=lat, mlp=moe)])


def model_numbers(size, batch, prompt, decode_steps, warmup):
    s, e = pairs.SIZES[size], conv_latent.SIZES[size]
    room = prompt + decode_steps + warmup + 64
    out = {}
    for name, make in (("memory_navulorn", lambda: build(memory_config(s), batch, room)), ("memory_balivik", lambda: build(balivik_mixers(s), batch, room)),
                       ("latent_navulorn", lambda: build(latent_config(e), batch, room)), ("latent_tusipel", lambda: conv_latent.build_tusipel(e, batch, room))):
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

    W, H, G, D, page = s["width"], s["heads"], s["kv_heads"], s["dim"], 64
    R, rot, win, chunk = ex["rank"], ex["rot"], ex["window"], ex["chunk"]
    nh, kD, kV = s["d_heads"], s["d_dim"], s["d_vdim"]
    E, k, F = ex["experts"], ex["top"], ex["ff"]
    rnd = lambda *shape, dt=bf: torch.randn(*shape, device=dev, dtype=dt)          # noqa: E731
    f32 = lambda *shape: torch.randn(*shape, device=dev)                           # noqa: E731
    for phase, T, ctx0 in (("prefill", prompt, 0), ("decode", 1, prompt)):
        B = batch
        N = B * T
        full = lambda v: torch.full((B,), v, dtype=torch.int32, device=dev)        # noqa: E731
        ctx, ql, lines = full(ctx0), full(T), torch.arange(B, dtype=torch.int32, device=dev)
        nblk = -(-(ctx0 + T) // page)
        table = torch.arange(B * nblk, dtype=torch.int32, device=dev).view(B, nblk)
        keys = ctx0 + T
        # embedding and stream
        ids = torch.randint(0, VOCAB, (B, T), device=dev, dtype=torch.int32)
        emb, big, prev = rnd(VOCAB, W), rnd(BIGRAM["buckets"] + 1, W), torch.zeros(B + 1, 1, dtype=torch.int32, device=dev)
        run(f"{phase}: bigram_embed (two table rows -> fp32 stream + bf16 copy, carried token)",
            lambda: ops.bigram_embed(ids, emb, big, 0.5, BIGRAM["mul_prev"], BIGRAM["mul_cur"], prev, lines, ctx, ql, bf), N * W * (2 + 2 + 4 + 2))
        x, y, w = f32(N, W), rnd(N, W), torch.ones(W, device=dev)
        run(f"{phase}: scaled_add_rmsnorm (sum + post-norm -> fp32 stream + bf16 copy)",
            lambda: ops.scaled_add_rmsnorm(x, y, w, 1.5, 1e-6, 0.0, bf), N * W * (4 + 2 + 4 + 2))
        run(f"{phase}: like: stream_add_rmsnorm (Sodudra / Tusipel: sum + pre-norm)",
            lambda: ops.stream_add_rmsnorm(x, (y,), weight=w, eps=1e-6, lp_dtype=bf), N * W * (4 + 2 + 4 + 2))
        # attention
        C = H * D + 2 * G * D
        p = rnd(B, T, C + H)
        cos, sin = f32(B, T, D // 2), f32(B, T, D // 2)
        kc, vc = rnd(B * nblk, page, G, D), rnd(B * nblk, page, G, D)
        qn, kn = torch.ones(H * D, device=dev), torch.ones(G * D, device=dev)
        run(f"{phase}: conv_qknorm_rope_append (row norms, rotate-half rotation, no convolution)",
            lambda: ops.conv_qknorm_rope_append(p, None, None, lines, ctx, ql, qn, kn, 1e-6, H, G, D, D, cos, sin, kc, vc, table, half=True), N * C * 2 * 2)
        cw, st = f32(C, 4), rnd(B + 1, 3, C)
        run(f"{phase}: like: conv_qknorm_rope_append (Fetodra: row norms, interleaved rotation, 4-tap convolution)",
            lambda: ops.conv_qknorm_rope_append(p, cw, st, lines, ctx, ql, qn, kn, 1e-6, H, G, D, D, cos, sin, kc, vc, table), N * C * 2 * 2)
        q, hg = rnd(B, T, H, D) * 0.2, p[..., C:]
        pairs_seen = B * sum(min(t + 1 + ctx0, chunk) for t in range(T))
        nb, fl = B * min(keys, T + chunk) * G * 2 * D * 2 + N * H * 2 * D * 2, 4.0 * pairs_seen * H * D
        run(f"{phase}: paged_window_attention ({H}/{G} heads of {D}, window {chunk}, gate per head)",
            lambda: ops.paged_window_attention(q, kc, vc, table, ctx, ql, 0.1, None, chunk, 0, hg, gate_per_head=True), nb, fl)
        run(f"{phase}: like: paged_window_attention (Zanivik: same window, no gate)",
            lambda: ops.paged_window_attention(q, kc, vc, table, ctx, ql, 0.1, None, chunk, 0), nb, fl)
        # latent attention
        Cq = H * (D + rot)
        pl, cache, lw = rnd(B, T, Cq + R + rot), rnd(B * nblk, page, 1, R + rot), torch.ones(R, device=dev)
        lc, ls = f32(B, T, rot // 2), f32(B, T, rot // 2)
        run(f"{phase}: latent_norm_append (latent norm, interleaved rotated key part)",
            lambda: ops.latent_norm_append(pl, Cq, R, lw, 1e-6, cache, table, ctx, ql, False, rot, lc, ls, interleaved=True), N * 2 * (R + rot) * 2)
        run(f"{phase}: like: latent_norm_append (Tusipel without query latent: rotate-half)",
            lambda: ops.latent_norm_append(pl, Cq, R, lw, 1e-6, cache, table, ctx, ql, False, rot, lc, ls), N * 2 * (R + rot) * 2)
        a = rnd(B, T, H, R + rot) * 0.2
        qs = pl.view(N, -1)[:, :Cq].unflatten(1, (H, D + rot)).view(B, T, H, D + rot)
        run(f"{phase}: rope_tail (interleaved, from the projection rows)", lambda: ops.rope_tail(qs, a, rot, lc, ls, True), N * H * rot * 2 * 2)
        qd = qs.contiguous()
        run(f"{phase}: like: rope_tail (Tusipel: rotate-half, dense queries)", lambda: ops.rope_tail(qd, a, rot, lc, ls), N * H * rot * 2 * 2)
        lat = 2.0 * B * H * (2 * R + rot) * sum(min(t + 1 + ctx0, win) for t in range(T))
        run(f"{phase}: paged_window_attention (latent rows of {R} + {rot}, window {win}; the same kernel in the Tusipel stack)",
            lambda: ops.paged_window_attention(a, cache, cache, table, ctx, ql, 0.1, None, win, 0, value_dim=R),
            B * min(keys, T + win) * (R + rot) * 2 + N * H * (2 * R + rot) * 2, lat)
        # matrix memory
        inner, qkv = nh * kV, nh * (2 * kD + kV)
        pm = rnd(B, T, -(-(qkv + inner + 2 * nh) // 8) * 8)
        ib, fb = torch.zeros(nh, device=dev), torch.full((nh,), 4.0, device=dev)
        S = torch.zeros(B + 1, nh, kV, kD, device=dev)
        NS = -(-kV // ops.MLSTM_SLICE)
        n_, m_ = torch.zeros(B + 1, nh, NS, kD, device=dev), torch.zeros(B + 1, nh, NS, device=dev)
        nb = N * (qkv * 2 + 4 * nh + inner * 4) + B * nh * kD * kV * 8
        run(f"{phase}: mlstm_scan ({nh} heads x {kD} x {kV}: gates, memory, denominators)",
            lambda: ops.mlstm_scan(pm, qkv + inner, ib, fb, GATE_CAP, S, n_, m_, lines, ctx, ql, nh, kD, kV), nb, flops=4.0 * N * nh * kD * kV, n=3)
        dec = torch.linspace(0.7, 0.999, nh, device=dev)
        run(f"{phase}: like: decay_scan (Balivik: fixed decays, SiLU)", lambda: ops.decay_scan(pm, dec, S, lines, ctx, ql, nh, kD, kV), nb,
            flops=4.0 * N * nh * kD * kV, n=3)
        o, wn, wh, gate = f32(B, T, inner), torch.ones(inner, device=dev), torch.ones(kV, device=dev), pm[..., qkv:qkv + inner]
        run(f"{phase}: head_rmsnorm_gate (weight per channel)", lambda: ops.head_rmsnorm_gate(o, wn, nh, 1e-6, gate, "sigmoid", bf), N * inner * 8)
        run(f"{phase}: like: head_rmsnorm_gate (Balivik: weight shared by the heads)", lambda: ops.head_rmsnorm_gate(o, wh, nh, 1e-6, gate, "sigmoid", bf), N * inner * 8)
        # feed-forwards
        xm, rw, rb = rnd(N, W), f32(E, W) * W ** -0.5, f32(E)
        run(f"{phase}: router_topk (bias, softmax over the chosen)", lambda: ops.router_topk(xm, rw, k, "softmax", True, True, bias=rb), N * W * 2 + E * W * 4,
            2.0 * N * W * E)
        run(f"{phase}: like: router_topk (Tusipel: softmax scores)", lambda: ops.router_topk(xm, rw, k, "softmax", False), N * W * 2 + E * W * 4, 2.0 * N * W * E)
        _, tw, ti = ops.router_topk(xm, rw, k, "softmax", True, True, bias=rb * 0)
        gu, dn = rnd(E, 2 * F, W) * 0.02, rnd(E, W, F) * 0.02
        used = min(E, N * k)
        run(f"{phase}: experts, SiLU (the same kernels in the Tusipel stack)", lambda: ops.moe_experts(xm, gu, dn, tw, ti, "silu_mul"),
            (used * 3 * F * W + N * W * 2) * 2, 6.0 * N * k * F * W)
        ff = s["ff"]
        wgu = rnd(2 * ff, W) * 0.02
        run(f"{phase}: dense gate and up projection, tanh GELU product in the epilogue", lambda: ops.linear(xm, wgu, act="gelu_tanh_mul"),
            (2 * ff * W + N * (W + ff)) * 2, 4.0 * N * ff * W)
        run(f"{phase}: like: dense gate and up projection, SiLU (Balivik)", lambda: ops.linear(xm, wgu, act="silu_mul"), (2 * ff * W + N * (W + ff)) * 2,
            4.0 * N * ff * W)
    return rows


def run(size="small", batch=4, prompt=1024, decode_steps=32, warmup=3):
    peaks = {}
    p = os.path.join(os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__)))), "MEASURED_PEAKS.json")
    if os.path.isfile(p):
        with open(p) as f:
            peaks = json.load(f)
    hbm, tf = float(peaks.get("hbm_gbs", 6650.0)), float(peaks.get("bf16_tflops", 1590.0))
    res = dict(size=size, shapes=pairs.SIZES[size], expert_shapes=conv_latent.SIZES[size], batch=batch, prompt=prompt, decode_steps=decode_steps,
               hbm_gbs=hbm, bf16_tflops=tf, peaks_source="measured" if peaks else "fallback")
    res.update(model_numbers(size, batch, prompt, decode_steps, warmup))
    res["kernels"] = kernel_table(size, batch, prompt, hbm, tf)
    return res
