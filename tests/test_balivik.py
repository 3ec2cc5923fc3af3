"""Balivik through the engine (loader, paged cache, state lines, ragged batches, scheduler) against the plain definition in
``balivik_oracle.py``.  Every test makes its own small configuration and random checkpoint; the CPU tests run the PyTorch
definitions of the ops in float32, the ``gpu`` tests the sm_100a kernels in float32 and bfloat16."""
import json
import os

import pytest
import torch

import balivik_oracle as oracle

PAGE = 8


def attn(heads=4, kv_heads=2, dim=12, vdim=10, rot=8, base=60.0, scale=0.3, diff=0.4):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, diff=diff)
    if rot:
        m["rot"] = dict(base=base, dims=rot)
    return m


def light(heads=3, dim=10, vdim=6, decay=(0.9, 0.5, 0.995)):
    return dict(heads=heads, dim=dim, vdim=vdim, decay=list(decay))


def delta(heads=4, kv_heads=2, dim=8, vdim=12, conv=3):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv)


def dense(ff=28):
    return dict(kind="dense", ff=ff)


def moe(experts=5, top=2, ff=14, limit=0.9):
    return dict(kind="moe", expert=dict(ff=ff, limit=limit), router=dict(experts=experts, top=top))


def layer(kind, mixer, mlp):
    return dict(type=kind, mixer=mixer, mlp=mlp)


def make_config(layers, width=36, vocab=83, eps=1e-4, streams=3, taps=3, loop=None, logit_scale=0.6):
    cfg = dict(architecture="Balivik", layers=layers, norm=dict(eps=eps), streams=streams, canon=dict(taps=taps), logit_scale=logit_scale,
               vocab=vocab, width=width)
    if loop:
        cfg["loop"] = dict(start=loop[0], stop=loop[1], times=loop[2])
    return cfg


STACK = [layer("channel_delta", delta(), moe()), layer("attention", attn(), dense()), layer("lightning", light(), None),
         layer("attention", attn(heads=3, kv_heads=3, dim=6, vdim=14, rot=6, diff=0.2), moe(experts=7, top=1, ff=9, limit=2.0))]
LOOP = (1, 3, 2)


def make_weights(cfg, seed=0, ranks=(5, 7)):
    """Random checkpoint in the design's tensor names (bf16-representable values), every part large enough to matter."""
    g = torch.Generator().manual_seed(seed)
    r = lambda *s, std=1.0, mean=0.0: (torch.randn(s, generator=g) * std + mean).bfloat16().float()       # noqa: E731
    W, V, S, w = cfg["width"], cfg["vocab"], cfg["streams"], {}
    w["embed"], w["head"], w["final.norm"] = r(V, W, std=0.7), r(V, W, std=W ** -0.5 * 3), r(std=0.1, mean=1.1)
    lin = lambda o, i, s=1.5: r(o, i, std=i ** -0.5 * s)       # noqa: E731
    for i, L in enumerate(cfg["layers"]):
        a, f, m = f"l{i}.", L["mlp"], L["mixer"]
        for q in (1, 2) if f is not None else (1,):
            w[f"{a}norm{q}"] = r(std=0.2, mean=1.0)
            w[f"{a}hc{q}.in"], w[f"{a}hc{q}.out"] = r(S, std=0.3, mean=1.0 / S), r(S, std=0.4, mean=0.8)
            w[f"{a}hc{q}.mix"] = (torch.eye(S) * 0.8 + r(S, S, std=0.25)).bfloat16().float()
        w[a + "canon1"] = r(W, cfg["canon"]["taps"], std=0.4)
        p, H, D, Dv = a + "mix.", m["heads"], m["dim"], m["vdim"]
        G = m.get("kv_heads", H)
        if L["type"] == "attention":
            w[p + "q"], w[p + "k"], w[p + "v"] = lin(2 * H * D, W), lin(2 * G * D, W), lin(G * Dv, W)
            for n in ("lq1", "lk1", "lq2", "lk2"):
                w[p + n] = r(D, std=0.35)
        elif L["type"] == "lightning":
            w[p + "q"], w[p + "k"], w[p + "v"], w[p + "g"] = lin(H * D, W), lin(H * D, W), lin(H * Dv, W), lin(H * Dv, W)
            w[p + "norm"] = r(H * Dv, std=0.3, mean=1.0)
        else:
            K = m["conv"]
            for n, rows in (("q", G * D), ("k", G * D), ("v", H * Dv)):
                w[p + n], w[p + n + ".conv"] = lin(rows, W), r(rows, K, std=0.6)
            w[p + "b"], w[p + "A_log"], w[p + "dt_bias"], w[p + "norm"] = lin(H, W), r(H, std=0.5, mean=-1.5), r(H * D, std=0.7), r(Dv, std=0.3, mean=1.0)
            w[p + "a1"], w[p + "a2"], w[p + "g1"], w[p + "g2"] = lin(ranks[0], W), lin(H * D, ranks[0]), lin(ranks[1], W), lin(H * Dv, ranks[1])
        w[p + "o"] = lin(W, H * Dv, 1.0)
        p = a + "mlp."
        if f is None:
            continue
        if f["kind"] == "dense":
            w[p + "gate"], w[p + "up"], w[p + "down"] = lin(f["ff"], W), lin(f["ff"], W), lin(W, f["ff"], 1.0)
        else:
            E, k, ff = f["router"]["experts"], f["router"]["top"], f["expert"]["ff"]
            for e in range(E):
                w[f"{p}e{e}.gate"], w[f"{p}e{e}.up"], w[f"{p}e{e}.down"] = lin(ff, W), lin(ff, W), lin(W, ff, 1.0)
            w[p + "table"] = torch.stack([torch.randperm(E, generator=g)[:k] for _ in range(V)]).int()
    return w


def make_engine(tmp_path, cfg, w, dtype="float32", device="cpu", max_tokens=512, max_requests=4, name="ckpt", page=PAGE):
    from safetensors.torch import save_file
    from neuronx_distributed_inference_b200.runtime.scheduler import build_engine
    d = tmp_path / name
    os.makedirs(d, exist_ok=True)
    with open(d / "config.json", "w") as f:
        json.dump(cfg, f)
    save_file({k: (v if v.dtype == torch.int32 else v.bfloat16()).contiguous() for k, v in w.items()}, str(d / "model.safetensors"))
    return build_engine(str(d), dtype, max_tokens, max_requests, page, device=device)


def rel_err(got, want):
    got, want = got.double(), want.double()
    return float((got - want).norm() / want.norm().clamp_min(1e-9))


def feed(engine, rid, tokens, cuts, want=None):
    rows, a = [], 0
    for b in list(cuts) + [len(tokens)]:
        if b <= a:
            continue
        idx = [i - a for i in (range(a, b) if want is None else [p for p in want if a <= p < b])]
        rows.append(engine.step([(rid, tokens[a:b], idx)])[0])
        a = b
    return torch.cat(rows, 0)


TOL = {"float32": 3e-4, "bfloat16": 8e-2}


def close(got, want, dtype):
    """float32: the whole block within a tight relative error.  bfloat16: in stacks this narrow a norm over a handful of channels, the
    difference of two maps or a peaked softmax can magnify the rounding of single positions, so positions are assessed one by one: the
    typical one within the tolerance, few beyond three times that."""
    if dtype == "float32":
        return rel_err(got, want) < TOL[dtype]
    got, want = got.double(), want.double()
    e = (got - want).norm(dim=-1) / want.norm(dim=-1).clamp_min(1e-9)
    return float(e.median()) < TOL[dtype] and float((e > 3 * TOL[dtype]).double().mean()) <= 0.1


def check_schedules(tmp_path, device, dtype, layers=STACK, T=61, seed=0, ranks=(5, 7), **cfg_kw):
    cfg_kw.setdefault("loop", LOOP if layers is STACK else None)
    cfg = make_config(layers, **cfg_kw)
    w = make_weights(cfg, seed, ranks)
    eng = make_engine(tmp_path, cfg, w, dtype, device)
    toks = torch.randint(0, cfg["vocab"], (T,), generator=torch.Generator().manual_seed(seed + 1)).tolist()
    want = oracle.forward(cfg, w, toks)
    whole = feed(eng, "whole", toks, [])
    assert close(whole, want, dtype)
    eng.release("whole")
    # most of the prompt at once, the rest token by token (slot and pages of the released request are used again): states, carried rows
    # and keys go on from where the prompt left them
    dec = feed(eng, "dec", toks, [T - 25] + list(range(T - 24, T)))
    assert close(dec, want, dtype) and close(dec[-25:], want[-25:], dtype)
    eng.release("dec")
    # token by token from the first token on
    one = feed(eng, "one", toks[:24], range(1, 24))
    assert close(one, want[:24], dtype) and close(one[:3], want[:3], dtype)
    eng.release("one")
    # portions of changing size, down to two tokens and across page borders
    cuts, a, sizes = [], 0, [2, 7, 2, 3, PAGE, 1, 2, 13, 5, 2]
    while a < T:
        a += sizes[len(cuts) % len(sizes)]
        cuts.append(min(a, T))
    ch = feed(eng, "ch", toks, cuts)
    assert close(ch, want, dtype)
    eng.release("ch")
    assert eng.pages.available == eng.pages.num_pages and eng.slots.available == eng.slots.num_pages
    return eng, cfg, w


def check_mixed_batches(eng, cfg, w, dtype, n_req=6, seed=3):
    """Unequal requests side by side (portions of some beside single tokens of others) against each alone; more requests than slots,
    so slots and pages are freed and taken again."""
    g = torch.Generator().manual_seed(seed)
    lens = [int(torch.randint(5, 60, (1,), generator=g)) for _ in range(n_req)]
    reqs = [torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for n in lens]
    want = [oracle.forward(cfg, w, r) for r in reqs]
    got, at = [[] for _ in reqs], [0] * n_req
    waiting, live, step = list(range(n_req)), [], 0
    while waiting or live:
        while waiting and len(live) < 4:
            live.append(waiting.pop(0))
        entries = []
        for k, i in enumerate(live):
            if len(live) > 1 and (step + 2 * k) % 5 == 4:
                continue                              # left out of this step, goes on later
            left = len(reqs[i]) - at[i]
            n = 1 if (at[i] > 0 and (step + k) % 3 == 0) else min(left, [2, 9, 4, 17][(step + i) % 4])
            entries.append((("r", i), reqs[i][at[i]:at[i] + n], list(range(n))))
        rows = eng.step(entries)
        for (rid, toks, _), row in zip(entries, rows):
            i = rid[1]
            got[i].append(row)
            at[i] += len(toks)
            if at[i] == len(reqs[i]):
                eng.release(rid)
                live.remove(i)
        step += 1
    if dtype == "float32":
        for i in range(n_req):
            assert close(torch.cat(got[i], 0), want[i], dtype), i
    else:
        assert close(torch.cat([torch.cat(x, 0) for x in got], 0), torch.cat(want, 0), dtype)
    for i in range(n_req):          # a request's rows do not depend on its neighbours: the same request fed alone
        alone = feed(eng, ("alone", i), reqs[i], [])
        eng.release(("alone", i))
        e = (torch.cat(got[i], 0).double() - alone.double()).norm(dim=-1) / want[i].norm(dim=-1)
        assert float(e.median()) < TOL[dtype] and float((e > 3 * TOL[dtype]).double().mean()) <= 0.1, i


def check_generate(eng, cfg, w, dtype):
    g = torch.Generator().manual_seed(11)
    prompts = [torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for n in (5, 23, 1, 40, 12, 9)]
    outs = eng.generate(prompts, max_new_tokens=6, max_step_tokens=16)
    for p, o in zip(prompts, outs):
        assert len(o) == 6
        seq = list(p)
        for tok in o:       # every emitted token is the arg-max of the plain model (ties aside: compare its logit with the best)
            lg = oracle.forward(cfg, w, seq)[-1]
            assert float(lg.max() - lg[tok]) <= (1e-3 if dtype == "float32" else 0.15) * float(lg.abs().max())
            seq.append(tok)


# ---- CPU: PyTorch definitions of the ops, float32 --------------------------------------------------------------------------
def test_stack_schedules_mixed_batches_and_generation(tmp_path):
    eng, cfg, w = check_schedules(tmp_path, "cpu", "float32")
    check_mixed_batches(eng, cfg, w, "float32")
    check_generate(eng, cfg, w, "float32")


OTHER = [
    # one layer of each kind alone: one head everywhere, one stream, one tap, no feed-forward
    ([layer("attention", attn(heads=1, kv_heads=1, dim=4, vdim=4, rot=4, diff=0.9), None)], dict(width=20, vocab=31, streams=1, taps=1)),
    ([layer("lightning", light(heads=1, dim=4, vdim=4, decay=(1.0,)), None)], dict(width=20, vocab=31, streams=2, taps=2)),
    ([layer("channel_delta", delta(heads=1, kv_heads=1, dim=4, vdim=4, conv=1), None)], dict(width=20, vocab=31, streams=2, taps=5, logit_scale=1.0)),
    # nothing rotated, one expert, every expert chosen, a loop over the whole stack, value size above key size, six taps
    ([layer("attention", attn(heads=6, kv_heads=1, dim=6, vdim=20, rot=0), moe(experts=1, top=1, limit=0.3)),
      layer("channel_delta", delta(heads=6, kv_heads=3, dim=20, vdim=4, conv=6), moe(experts=3, top=3, ff=6))], dict(width=28, streams=4, taps=4, loop=(0, 2, 3))),
    # sizes that coincide (head, value and state sizes, heads and kv heads), a loop that runs once, a span at the end
    ([layer("channel_delta", delta(heads=2, kv_heads=2, dim=8, vdim=8, conv=2), dense(32)), layer("lightning", light(heads=2, dim=8, vdim=8, decay=(0.25, 0.0)), dense(32)),
      layer("attention", attn(heads=2, kv_heads=2, dim=8, vdim=8, rot=8), dense(32))], dict(width=32, streams=2, taps=2, loop=(2, 3, 1))),
    # odd sizes: width, keys, values and streams that no vector access divides
    ([layer("channel_delta", delta(heads=3, kv_heads=1, dim=7, vdim=5, conv=4), moe(experts=4, top=2, ff=7)), layer("lightning", light(heads=3, dim=9, vdim=7), dense(13)),
      layer("attention", attn(heads=3, kv_heads=1, dim=10, vdim=7, rot=2), None)], dict(width=35, streams=5, taps=8, loop=(0, 1, 2))),
]


@pytest.mark.parametrize("layers,kw", OTHER)
def test_other_sizes_and_layouts(tmp_path, layers, kw):
    check_schedules(tmp_path, "cpu", "float32", layers=layers, T=45, seed=5, ranks=(3, 2), **kw)


def _model(eng):
    return eng.app.context_encoding_model.model if hasattr(eng.app, "context_encoding_model") else eng.app.model


def check_streams(tmp_path, device, tol):
    cfg = make_config(STACK, loop=LOOP)
    w = make_weights(cfg, 2)
    eng = make_engine(tmp_path, cfg, w, device=device)
    toks = list(range(3, 20))
    streams = []
    oracle.forward(cfg, w, toks, streams)
    T = len(toks)
    on = lambda t: t.to(device)       # noqa: E731
    out = _model(eng)(on(torch.tensor([toks])), attention_mask=on(torch.ones(1, T, dtype=torch.int32)), position_ids=on(torch.arange(T).view(1, T)),
                      seq_ids=on(torch.tensor([0])), slot_mapping=on(torch.arange(T).view(1, T).int()), block_table=on(torch.arange(4).view(1, 4).int()),
                      computed_context_lens=torch.tensor([0]), capture=True)
    assert len(streams) == 6
    for i, s in enumerate(streams):
        assert float((out.captured[f"runs.{i}.out"][0].double().cpu() - s).abs().max() / s.abs().max()) < tol, i


def test_streams_after_every_layer_run(tmp_path):
    check_streams(tmp_path, "cpu", 5e-5)


def test_long_decoding_over_many_pages(tmp_path):
    cfg = make_config(STACK[:2])
    w = make_weights(cfg, 9)
    eng = make_engine(tmp_path, cfg, w)
    toks = torch.randint(0, cfg["vocab"], (90,), generator=torch.Generator().manual_seed(2)).tolist()
    got = feed(eng, "x", toks, range(3, 90))         # 3-token prompt, then 87 single tokens over twelve pages
    assert rel_err(got, oracle.forward(cfg, w, toks)) < TOL["float32"]


def test_cache_pool_smaller_than_all_requests(tmp_path):
    """The pool holds two requests' worth of pages: the third request runs on the pages and the slot the first gave back, and must not
    see what the first left in them (keys, carried rows, convolution tails, recurrent states)."""
    cfg = make_config(STACK, loop=LOOP)
    w = make_weights(cfg, 4)
    eng = make_engine(tmp_path, cfg, w, max_tokens=64, max_requests=2)
    g = torch.Generator().manual_seed(6)
    reqs = [torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for n in (30, 27, 31)]
    a = feed(eng, 0, reqs[0], [11])
    b = feed(eng, 1, reqs[1], [5, 6])
    with pytest.raises(MemoryError):
        eng.step([(2, reqs[2], [])])
    eng.release(2)
    eng.release(0)
    c = feed(eng, 2, reqs[2], [2, 17])
    for got, r in ((a, reqs[0]), (b, reqs[1]), (c, reqs[2])):
        assert rel_err(got, oracle.forward(cfg, w, r)) < TOL["float32"]


def check_long_lived_states(tmp_path, device):
    """Decays close to one: what the first tokens wrote into the recurrent states still shapes the logits hundreds of tokens on, whether the
    prompt arrives whole, in portions or token by token."""
    cfg = make_config([layer("channel_delta", delta(), None), layer("lightning", light(decay=(0.999, 1.0, 0.99)), None)])
    w = make_weights(cfg, 1)
    w["l0.mix.A_log"].fill_(-9.0)
    eng = make_engine(tmp_path, cfg, w, device=device, max_tokens=1024)
    g = torch.Generator().manual_seed(8)
    toks = torch.randint(0, cfg["vocab"], (260,), generator=g).tolist()
    other = [(toks[0] + 1) % cfg["vocab"], (toks[1] + 7) % cfg["vocab"]] + toks[2:]
    want, moved = oracle.forward(cfg, w, toks), oracle.forward(cfg, w, other)
    assert rel_err(moved[-5:], want[-5:]) > 2e-3                  # the first two tokens matter at the end
    last = list(range(255, 260))
    for cuts in ([], [100, 200], [3] + list(range(230, 260))):
        got = feed(eng, "s", toks, cuts, want=last)
        eng.release("s")
        assert rel_err(got, want[-5:]) < TOL["float32"]


def test_a_long_lived_state_carries_the_first_tokens_far(tmp_path):
    check_long_lived_states(tmp_path, "cpu")


# ---- mechanisms alone: op definitions (CPU) or kernels (GPU) against the plain functions ---------------------------------------
def i32(dev, *x):
    return torch.tensor(x).int().to(dev)


def paged(rows, page, g, spare=3):
    """rows [n, G, C] -> (cache [blocks, page, G, C] on scattered pages, block table [1, blocks])."""
    n, G, C = rows.shape
    nblk = -(-n // page)
    perm = torch.randperm(nblk + spare, generator=g)[:nblk]
    cache = torch.zeros(nblk + spare, page, G, C)
    for j in range(n):
        cache[perm[j // page], j % page] = rows[j]
    return cache, perm.view(1, -1).int()


def loud_key_case(dev, dtype, target, pos, loud_map, *, page=4, as_prompt=False, extra=0, D=8, Dv=6):
    """Four heads over two kv heads; in map ``loud_map`` the key row ``target`` is made to dominate the query at ``pos`` (one query and one
    key are scaled so that one score stands out), in the other map the row ``pos`` itself.  Returns (op output, plain output, what the
    heads give when the target is seen) for the query at ``pos``."""
    from neuronx_distributed_inference_b200 import ops
    H, G, lam, diff, eps = 4, 2, 0.7, 0.25, 1e-5
    g = torch.Generator().manual_seed(target * 131 + pos)
    n = pos + 1 + extra
    k, v, q = torch.randn(n, G, 2, D, generator=g) * 0.1, torch.randn(n, G, Dv, generator=g), torch.randn(n, H, 2, D, generator=g) * 0.1
    if target < n:
        k[target, :, loud_map] = 6.0 / D ** 0.5 * 1.4
    k[pos, :, 1 - loud_map] = 6.0 / D ** 0.5 * 1.4
    q[pos] = 6.0 / D ** 0.5 * 1.4
    want = oracle.differential_attention(q[:pos + 1].double(), k[:pos + 1].double(), v[:pos + 1].double(), 0.4, lam, diff, eps)[pos].reshape(-1)
    kc, table = paged(k.view(n, 2 * G, D), page, torch.Generator().manual_seed(5))
    vc, _ = paged(v, page, torch.Generator().manual_seed(5))
    to = lambda t: t.to(dev, dtype)                                      # noqa: E731
    args = (0.4, torch.tensor([lam]).to(dev), 1.0 - diff, eps)
    qf = q.view(n, 2 * H, D)
    if as_prompt:
        got = ops.paged_diff_attention(to(qf.view(1, n, 2 * H, D)), to(kc), to(vc), table.to(dev), i32(dev, 0), i32(dev, n), *args)[0, pos]
    else:
        got = ops.paged_diff_attention(to(qf[pos].view(1, 1, 2 * H, D)), to(kc), to(vc), table.to(dev), i32(dev, pos), i32(dev, 1), *args)
    seen = v[min(target, n - 1)].double()
    o = seen - lam * v[pos].double() if loud_map == 0 else v[pos].double() - lam * seen
    row = (oracle.rms_norm(o, eps) * (1 - diff)).repeat_interleave(H // G, 0).reshape(-1).float()
    return got.float().cpu().view(-1), want.float(), row


# (position, loud key): far keys, page borders (pages of 4), the first tokens, the query itself
PLACES = [(300, 0), (301, 150), (300, 299), (0, 0), (4, 4), (8, 7), (8, 8), (64, 63), (64, 1), (40, 3)]


@pytest.mark.parametrize("pos,target", PLACES)
@pytest.mark.parametrize("as_prompt", [False, True])
def test_loud_keys_near_and_far_in_either_map(pos, target, as_prompt):
    for m in (0, 1):
        got, want, row = loud_key_case("cpu", torch.float32, target, pos, m, as_prompt=as_prompt)
        assert torch.allclose(got, want, atol=1e-4)
        assert torch.allclose(got, row, atol=2e-2)          # the loud row's value enters with the sign of its map


def test_a_prompt_does_not_see_later_rows_of_its_portion():
    got, want, row = loud_key_case("cpu", torch.float32, 21, 20, 0, as_prompt=True, extra=3)       # the loud row is one step ahead
    assert torch.allclose(got, want, atol=1e-4) and not torch.allclose(got, row, atol=0.3)


def ragged_case(B=3, T=11):
    return torch.tensor([0, 5, 40]).int(), torch.tensor([T, 4, 1]).int(), torch.tensor([2, 0, 3]).int()


def check_stream_mix(dev, dt, tol):
    """Write-back, mixing, read, norm (one number, a vector, none) and convolution, on ragged rows with carried rows; equal streams; no
    write-back; the carried rows advanced by portions of every size (also across several tiles of a row)."""
    from neuronx_distributed_inference_b200 import ops
    g = torch.Generator().manual_seed(0)
    rn = lambda *s: torch.randn(*s, generator=g)        # noqa: E731
    eps = 1e-3
    on = lambda t: None if t is None else t.to(dev)      # noqa: E731
    for W, S, K, T in ((36, 3, 3, 29), (64, 2, 4, 40), (35, 5, 8, 21), (1024, 4, 2, 11), (2304, 1, 4, 9), (32, 2, 1, 7), (5120, 2, 3, 6)):
        B = 2
        x, y = rn(B, T, S, W), rn(B, T, W).to(dt)
        mix, ow, iw, nw = rn(S, S), rn(S), rn(S), (rn(1) if K % 2 else rn(W))
        cw = rn(W, K) * 0.5
        xs = torch.einsum("btsw,sd->btdw", x.double(), mix.double()) + ow.double().view(1, 1, S, 1) * y.double().unsqueeze(2)
        h = oracle.rms_norm(torch.einsum("btsw,s->btw", xs, iw.double()), eps, nw.double())
        want = torch.stack([h[b] + oracle.causal_conv(h[b], cw.double()) for b in range(B)])
        state = (rn(5, K - 1, W) * 9).to(dev) if K > 1 else None          # what earlier requests left in the lines
        args = (on(mix), on(ow), on(iw), on(nw), on(cw), state)
        xn, r = ops.stream_mix_norm_conv(on(x), on(y), *args, i32(dev, 3, 1), i32(dev, 0, 0), i32(dev, T, T), eps, dt)
        assert torch.allclose(xn.double().cpu(), xs, atol=1e-4, rtol=1e-5)
        assert torch.allclose(r.double().cpu(), want, atol=tol * 8, rtol=tol)
        if K > 1:
            keep = torch.cat([torch.zeros(B, K - 1, W, dtype=torch.float64), h], 1)[:, T:]
            assert torch.allclose(state[3].double().cpu(), keep[0], atol=1e-4) and torch.allclose(state[1].double().cpu(), keep[1], atol=1e-4)
        # the same rows in unequal portions
        at, rows, step = [0, 0], [[], []], 0
        while min(at) < T:
            n = [min(T - at[b], [1, 2, 5, 12][(step + b) % 4]) for b in range(B)]
            m = max(n)
            xp, yp = torch.zeros(B, m, S, W), torch.zeros(B, m, W, dtype=dt)
            for b in range(B):
                xp[b, :n[b]], yp[b, :n[b]] = x[b, at[b]:at[b] + n[b]], y[b, at[b]:at[b] + n[b]]
            _, r = ops.stream_mix_norm_conv(on(xp), on(yp), *args, i32(dev, 0, 4), i32(dev, *at), i32(dev, *n), eps, dt)
            for b in range(B):
                rows[b].append(r[b, :n[b]].double().cpu())
                at[b] += n[b]
            step += 1
        for b in range(B):
            assert torch.allclose(torch.cat(rows[b]), want[b], atol=tol * 8, rtol=tol)
        # equal streams, no write-back, no norm
        e = x[:, :, 0].contiguous()
        same, r = ops.stream_mix_norm_conv(on(e), None, None, None, on(iw), None, None, None, None, None, None, eps)
        assert torch.allclose(r.double().cpu(), e.double() * iw.double().sum(), atol=1e-4) and same.shape == e.shape
        xn, r = ops.stream_mix_norm_conv(on(e), on(y), on(mix), on(ow), on(iw), on(nw), None, None, None, None, i32(dev, T, 2), eps, dt)
        xs = torch.einsum("btsw,sd->btdw", e.double().unsqueeze(2).expand(-1, -1, S, -1), mix.double()) + ow.double().view(1, 1, S, 1) * y.double().unsqueeze(2)
        assert torch.allclose(xn[0].double().cpu(), xs[0], atol=1e-4, rtol=1e-5) and torch.allclose(xn[1, :2].double().cpu(), xs[1, :2], atol=1e-4, rtol=1e-5)


def check_rope_append_shared_values(dev, dt, tol):
    """Rotation of both maps and the cache rows when two key heads share one value head; positions from the context length."""
    from neuronx_distributed_inference_b200 import ops
    g = torch.Generator().manual_seed(1)
    rn = lambda *s: torch.randn(*s, generator=g)        # noqa: E731
    B, T, page, nblk = 3, 11, 4, 14
    ctx, ql, _ = ragged_case(B, T)
    for H, G, D, Dv, R in ((4, 2, 12, 10, 8), (2, 1, 64, 128, 32), (3, 3, 10, 7, 2), (2, 2, 16, 16, 0), (1, 1, 128, 64, 128)):
        C = 2 * H * D + 2 * G * D + G * Dv
        p = rn(B, T, C + 16).to(dt)[..., 8:8 + C]
        rot = dict(base=77.0, dims=R)
        table = torch.randperm(B * nblk, generator=g).view(B, nblk).int()
        kd, vd = torch.zeros(B * nblk, page, 2 * G, D, dtype=dt).to(dev), torch.zeros(B * nblk, page, G, Dv, dtype=dt).to(dev)
        cos = sin = None
        if R:
            f = torch.tensor([77.0 ** (-2.0 * i / R) for i in range(R // 2)], dtype=torch.float64)
            ang = (ctx.double().view(B, 1) + torch.arange(T).double().view(1, T)).unsqueeze(-1) * f
            cos, sin = torch.cos(ang).float().to(dev), torch.sin(ang).float().to(dev)
        q = ops.head_norm_rope_append(p.to(dev), 2 * H, 2 * G, D, Dv, cos, sin, None, None, 0, 1e-3, False, kd, vd, table.to(dev), ctx.to(dev), ql.to(dev), n_v=G)
        for b in range(B):
            n, c0 = int(ql[b]), int(ctx[b])
            rows = p[b, :n].double()
            assert torch.allclose(q[b, :n].double().cpu(), oracle.rotate(rows[:, :2 * H * D].view(n, 2 * H, D), rot, c0), atol=tol * 3, rtol=tol)
            kw = oracle.rotate(rows[:, 2 * H * D:2 * (H + G) * D].view(n, 2 * G, D), rot, c0)
            for t in range(n):
                at = (int(table[b, (c0 + t) // page]), (c0 + t) % page)
                assert torch.allclose(kd[at].double().cpu(), kw[t], atol=tol * 3, rtol=tol)
                assert torch.equal(vd[at].double().cpu(), rows[t, 2 * (H + G) * D:].view(G, Dv))


def check_channel_delta(dev, dt, tol):
    """Rows and recurrence against the plain loop: whole rows and unequal portions with carried rows and state; heads that share q / k
    heads; lines used in another order; decays near one and near zero."""
    from neuronx_distributed_inference_b200 import ops
    g = torch.Generator().manual_seed(2)
    rn = lambda *s: torch.randn(*s, generator=g)        # noqa: E731
    on = lambda t: t.to(dev)      # noqa: E731
    for H, G, D, Dv, T, K in ((4, 2, 8, 10, 37, 3), (3, 1, 7, 5, 20, 8), (2, 2, 16, 20, 18, 1), (2, 1, 128, 16, 40, 4), (1, 1, 136, 8, 35, 2), (2, 1, 64, 36, 33, 4)):
        B, C = 2, 2 * G * D + H * Dv
        p = rn(B, T, C + H + 3).to(dt)
        a = (rn(B, T, H * D + 4) * 2).to(dt)[..., :H * D]
        cw, A_log, dtb = rn(C, K) * 0.6, rn(H) * 1.5 - 1.0, rn(H * D)
        conv = torch.stack([oracle.silu(oracle.causal_conv(p[b, :, :C].double(), cw.double())) for b in range(B)])
        q = (oracle.unit(conv[..., :G * D].reshape(B, T, G, D)) * D ** -0.5).repeat_interleave(H // G, 2)
        k = oracle.unit(conv[..., G * D:2 * G * D].reshape(B, T, G, D)).repeat_interleave(H // G, 2)
        beta = torch.sigmoid(p[..., C:C + H].double())
        decay = torch.exp(-torch.exp(A_log.double()).view(1, 1, H, 1) * oracle.softplus(a.double() + dtb.double()).view(B, T, H, D))
        want = torch.stack([oracle.channel_delta_rule(q[b], k[b], conv[b, :, 2 * G * D:].reshape(T, H, Dv), beta[b], decay[b]) for b in range(B)]).reshape(B, T, -1)

        def run(rows, arows, lines, ctx, ql, cst, sst):
            where = (i32(dev, *lines), i32(dev, *ctx), i32(dev, *ql))
            pr = on(rows)
            f = ops.delta_front(pr, pr[..., C:C + H], on(arows), on(cw), on(A_log), on(dtb), cst, *where, H, G, D, Dv)
            return ops.channel_delta_scan(*f, sst, *where, H, G, D, Dv)
        fresh = lambda: ((rn(5, K - 1, C) * 9).to(dt).to(dev), (rn(5, H, Dv, D) * 9).to(dev))       # noqa: E731  (left by earlier requests)
        cst, sst = fresh()
        got = run(p, a, (3, 1), (0, 0), (T, T), cst, sst)
        assert torch.allclose(got.double().cpu(), want, atol=tol, rtol=tol)
        cst2, sst2 = fresh()
        at, rows, step = [0, 0], [[], []], 0
        while min(at) < T:
            n = [min(T - at[b], [1, 2, 19, 5][(step + b) % 4]) for b in range(B)]
            m = max(n)
            pp, ap = torch.zeros(B, m, p.shape[2], dtype=dt), torch.zeros(B, m, H * D, dtype=dt)
            for b in range(B):
                pp[b, :n[b]], ap[b, :n[b]] = p[b, at[b]:at[b] + n[b]], a[b, at[b]:at[b] + n[b]]
            y = run(pp, ap, (0, 4), at, n, cst2, sst2)
            for b in range(B):
                rows[b].append(y[b, :n[b]].double().cpu())
                at[b] += n[b]
            step += 1
        for b in range(B):
            assert torch.allclose(torch.cat(rows[b]), want[b], atol=tol, rtol=tol)
        assert torch.equal(cst2[0].cpu(), cst[3].cpu()) and torch.equal(cst2[4].cpu(), cst[1].cpu())
        assert torch.allclose(sst2[0].cpu(), sst[3].cpu(), atol=tol, rtol=tol) and torch.allclose(sst2[4].cpu(), sst[1].cpu(), atol=tol, rtol=tol)


def check_decay_scan(dev, dt, tol):
    """Fixed decays from 0 to 1 against the plain loop, whole rows and unequal portions, then the gated norm over all heads."""
    from neuronx_distributed_inference_b200 import ops
    g = torch.Generator().manual_seed(3)
    rn = lambda *s: torch.randn(*s, generator=g)        # noqa: E731
    on = lambda t: t.to(dev)      # noqa: E731
    for H, D, Dv, T in ((3, 10, 6, 37), (2, 7, 5, 18), (4, 64, 64, 150), (2, 128, 128, 200), (2, 64, 128, 65), (4, 128, 64, 129), (1, 136, 20, 35), (2, 32, 48, 64), (2, 16, 16, 70)):
        B, C = 2, H * (2 * D + Dv)
        p = rn(B, T, C + H * Dv).to(dt)
        decay = torch.tensor([0.999, 0.5, 1.0, 0.0][:H]) if H > 1 else torch.tensor([0.97])
        x = oracle.silu(p[..., :C].double())
        q, k, v = (t.reshape(B, T, H, -1) for t in x.split([H * D, H * D, H * Dv], -1))
        want = torch.stack([oracle.decayed_outer_products(q[b], k[b], v[b], decay.double()) for b in range(B)]).reshape(B, T, -1)
        big = float(want.abs().max())
        st = (rn(5, H, Dv, D) * 9).to(dev)
        y = ops.decay_scan(on(p), on(decay), st, i32(dev, 3, 1), i32(dev, 0, 0), i32(dev, T, T), H, D, Dv)
        assert torch.allclose(y.double().cpu() / big, want / big, atol=tol, rtol=tol)
        st2 = (rn(5, H, Dv, D) * 9).to(dev)
        at, rows, step = [0, 0], [[], []], 0
        while min(at) < T:
            n = [min(T - at[b], [1, 2, 19, 70][(step + b) % 4]) for b in range(B)]
            m = max(n)
            pp = torch.zeros(B, m, p.shape[2], dtype=dt)
            for b in range(B):
                pp[b, :n[b]] = p[b, at[b]:at[b] + n[b]]
            yy = ops.decay_scan(on(pp), on(decay), st2, i32(dev, 0, 4), i32(dev, *at), i32(dev, *n), H, D, Dv)
            for b in range(B):
                rows[b].append(yy[b, :n[b]].double().cpu())
                at[b] += n[b]
            step += 1
        for b in range(B):
            assert torch.allclose(torch.cat(rows[b]) / big, want[b] / big, atol=tol, rtol=tol)
        assert torch.allclose(st2[0].cpu(), st[3].cpu(), atol=tol * big, rtol=tol) and torch.allclose(st2[4].cpu(), st[1].cpu(), atol=tol * big, rtol=tol)
        wn = rn(H * Dv)
        gate = on(p)[..., C:]
        o = ops.group_rmsnorm(y, on(wn), 1, 1e-3, out_dtype=dt, gate=gate, act="sigmoid")
        o_want = oracle.rms_norm(y.double().cpu(), 1e-3, wn.double()) * torch.sigmoid(p[..., C:].double())
        otol = 1e-2 if dt == torch.bfloat16 else 2e-5
        assert torch.allclose(o.double().cpu(), o_want, atol=otol, rtol=otol)


def check_table_experts(dev, dt, tol):
    """Routing by token id (padding routed nowhere) and the clamped gate product with a limit that bites, for a handful of tokens and many."""
    from neuronx_distributed_inference_b200 import ops
    g = torch.Generator().manual_seed(4)
    rn = lambda *s: torch.randn(*s, generator=g)        # noqa: E731
    for W, I, E, k, limit in ((36, 14, 5, 2, 0.8), (64, 64, 6, 3, 1.3), (128, 192, 4, 1, 0.4)):
        gu, dn = (rn(E, 2 * I, W) * W ** -0.5 * 2).to(dt), (rn(E, W, I) * I ** -0.5).to(dt)
        table = torch.stack([torch.randperm(E, generator=g)[:k] for _ in range(40)]).int()
        for B, T, ql in ((2, 3, (3, 1)), (2, 90, (90, 41))):
            ids = torch.randint(0, 40, (B, T), generator=g)
            x = (rn(B, T, W) * 1.5).to(dt)
            w, idx = ops.table_route(table.to(dev), ids.to(dev), i32(dev, *ql))
            y = ops.moe_experts(x.view(-1, W).to(dev), gu.to(dev), dn.to(dev), w, idx, "clamped_glu", act_params=(limit, 1.702)).view(B, T, W)
            ww = {f"e{e}.{n}": m[e].double() for n, m in (("gate", gu[:, :I]), ("up", gu[:, I:]), ("down", dn)) for e in range(E)}
            ww["table"] = table
            for b in range(B):
                want = oracle.table_moe(x[b, :ql[b]].double(), ids[b].tolist()[:ql[b]], dict(expert=dict(limit=limit)), ww, "")
                assert torch.allclose(y[b, :ql[b]].double().cpu(), want, atol=tol * 3, rtol=tol)
                assert not y[b, ql[b]:].any()


def test_stream_mixing_norm_and_convolution():
    check_stream_mix("cpu", torch.float32, 1e-5)


def test_rotation_and_cache_rows_with_shared_values():
    check_rope_append_shared_values("cpu", torch.float32, 1e-5)


def test_channel_delta_rule_and_what_it_carries():
    check_channel_delta("cpu", torch.float32, 2e-5)


def test_fixed_decays_and_their_carried_state():
    check_decay_scan("cpu", torch.float32, 1e-5)


def test_table_routing_and_clamped_experts():
    check_table_experts("cpu", torch.float32, 1e-5)


def test_lambda_is_folded_from_its_four_vectors():
    from neuronx_distributed_inference_b200.modules.attention.differential_attention import differential_lambda
    g = torch.Generator().manual_seed(0)
    v = [torch.randn(12, generator=g) * 0.3 for _ in range(4)]
    assert abs(float(differential_lambda(*v, 0.35)) - oracle.lambda_of(v[0], v[1], v[2], v[3], 0.35)) < 1e-6


def test_ranks_come_from_the_tensors(tmp_path):
    for name, ranks in (("a", (5, 7)), ("b", (9, 3))):
        cfg = make_config(STACK[:1])
        eng = make_engine(tmp_path, cfg, make_weights(cfg, 0, ranks), name=name)
        m = _model(eng).layers[0].mixer
        assert m.ranks == sum(ranks) and tuple(m.low_rank_up.weight.shape) == (4 * 8 + 4 * 12, sum(ranks))


def test_registry_picks_the_model_from_config_json(tmp_path):
    from neuronx_distributed_inference_b200.utils.constants import get_model_cls, model_type_of
    with open(tmp_path / "config.json", "w") as f:
        json.dump(make_config(STACK), f)
    assert get_model_cls(model_type_of(str(tmp_path))).__name__ == "NeuronBalivikForCausalLM"


def test_command_line_generates_from_token_ids(tmp_path, capsys):
    from neuronx_distributed_inference_b200 import inference_demo
    cfg = make_config(STACK, loop=LOOP)
    w = make_weights(cfg)
    eng = make_engine(tmp_path, cfg, w)
    want = eng.generate([[1, 2, 3, 4], [7, 8]], 5)
    inference_demo.main(["--model-type", "balivik", "--task-type", "causal-lm", "run", "--model-path", str(tmp_path / "ckpt"),
                         "--compiled-model-path", str(tmp_path / "c"), "--on-cpu", "--torch-dtype", "float32", "--prompt-token-ids", "1,2,3,4",
                         "--prompt-token-ids", "7,8", "--max-new-tokens", "5", "--pa-block-size", str(PAGE)])
    out = capsys.readouterr().out
    assert "Output 0: " + ",".join(map(str, want[0])) in out and "Output 1: " + ",".join(map(str, want[1])) in out


# ---- GPU: the sm_100a kernels --------------------------------------------------------------------------------------------------
@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_gpu_stack_schedules_mixed_batches_and_generation(tmp_path, dtype):
    from neuronx_distributed_inference_b200 import ops
    ops.stats.clear()
    eng, cfg, w = check_schedules(tmp_path, "cuda", dtype)
    check_mixed_batches(eng, cfg, w, dtype)
    check_generate(eng, cfg, w, dtype)
    for k in ("stream_mix_norm_conv", "head_norm_rope_append", "paged_diff_attention", "delta_front", "channel_delta_scan", "head_rmsnorm_gate",
              "decay_scan", "group_rmsnorm", "table_route", "gated_act_mul"):
        assert ops.stats[k] > 0, k
    tkg = eng.app.token_generation_model          # single-token steps replayed from CUDA graphs (capture did not fall back to eager)
    assert tkg.use_graphs and len(tkg._graphs) > 0


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_gpu_wider_stack(tmp_path, dtype):
    """Head sizes of 64 and 128 (tensor-core attention and chunked recurrence on bf16 portions, grouped expert GEMMs) beside sizes that take
    the CUDA-core kernels; recurrent heads with 128 and 136 key channels."""
    layers = [layer("attention", attn(heads=4, kv_heads=2, dim=64, vdim=128, rot=32, scale=0.12), moe(experts=6, top=2, ff=128, limit=1.1)),
              layer("channel_delta", delta(heads=4, kv_heads=2, dim=128, vdim=32, conv=4), dense(256)),
              layer("lightning", light(heads=2, dim=64, vdim=64, decay=(0.9, 0.998)), moe(experts=5, top=1, ff=64, limit=0.7)),
              layer("channel_delta", delta(heads=2, kv_heads=1, dim=136, vdim=20, conv=3), None),
              layer("attention", attn(heads=2, kv_heads=1, dim=128, vdim=64, rot=128, scale=0.09), dense(192))]
    eng, cfg, w = check_schedules(tmp_path, "cuda", dtype, layers=layers, T=77, width=256, vocab=301, eps=1e-6, seed=7, streams=2, taps=4, loop=(1, 4, 2), ranks=(24, 40))
    check_mixed_batches(eng, cfg, w, dtype, n_req=5)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("layers,kw", OTHER)
def test_gpu_other_sizes_and_layouts(tmp_path, dtype, layers, kw):
    check_schedules(tmp_path, "cuda", dtype, layers=layers, T=45, seed=5, ranks=(3, 2), **kw)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("pos,target", PLACES)
@pytest.mark.parametrize("as_prompt", [False, True])
@pytest.mark.parametrize("D,Dv", [(8, 6), (64, 128), (128, 64)])
def test_gpu_loud_keys_near_and_far_in_either_map(pos, target, dtype, as_prompt, D, Dv):
    for m in (0, 1):
        got, want, row = loud_key_case("cuda", dtype, target, pos, m, as_prompt=as_prompt, D=D, Dv=Dv)
        assert torch.allclose(got, want, atol=2e-4 if dtype == torch.float32 else 4e-2)
        assert torch.allclose(got, row, atol=6e-2)


@pytest.mark.gpu
def test_gpu_prompt_portions_over_a_prefix_match_the_plain_maps():
    """Tensor-core portions that start behind a cached prefix, several query blocks and key tiles, unequal rows of one batch."""
    from neuronx_distributed_inference_b200 import ops
    g = torch.Generator().manual_seed(9)
    H, G, page, lam, diff = 4, 2, 16, 0.6, 0.3
    for D, Dv in ((64, 64), (64, 128), (128, 128), (40, 72)):
        ctx, ql, T, nblk = (37, 0, 130), (100, 61, 1), 100, 16
        k, v = torch.randn(3, 240, G, 2, D, generator=g), torch.randn(3, 240, G, Dv, generator=g)
        q = torch.randn(3, T, H, 2, D, generator=g)
        kc, vc = torch.zeros(3 * nblk, page, 2 * G, D), torch.zeros(3 * nblk, page, G, Dv)
        table = torch.randperm(3 * nblk, generator=g).view(3, nblk).int()
        for b in range(3):
            for j in range(ctx[b] + ql[b]):
                kc[table[b, j // page], j % page], vc[table[b, j // page], j % page] = k[b, j].view(2 * G, D), v[b, j]
        for dt, tol in ((torch.float32, 2e-4), (torch.bfloat16, 5e-2)):
            to = lambda t: t.to("cuda", dt)                                      # noqa: E731
            got = ops.paged_diff_attention(to(q.view(3, T, 2 * H, D)), to(kc), to(vc), table.cuda(), i32("cuda", *ctx), i32("cuda", *ql), D ** -0.5,
                                           torch.tensor([lam]).cuda(), 1.0 - diff, 1e-5).double().cpu()
            rd = lambda t: t.to(dt).double()                                     # noqa: E731
            for b in range(3):
                n = ctx[b] + ql[b]
                full = torch.cat([torch.zeros(ctx[b], H, 2, D, dtype=torch.float64), rd(q[b, :ql[b]])])
                want = oracle.differential_attention(full, rd(k[b, :n]), rd(v[b, :n]), D ** -0.5, lam, diff, 1e-5)[ctx[b]:].reshape(ql[b], -1)
                e = (got[b, :ql[b]] - want).norm(dim=-1) / want.norm(dim=-1)
                assert float(e.max()) < tol and not got[b, ql[b]:].any(), (D, Dv, dt, b)


@pytest.mark.gpu
@pytest.mark.parametrize("dt,tol", [(torch.float32, 2e-5), (torch.bfloat16, 1e-2)])
def test_gpu_kernels_match_the_plain_functions(dt, tol):
    check_stream_mix("cuda", dt, tol)
    check_rope_append_shared_values("cuda", dt, tol)
    check_channel_delta("cuda", dt, 1e-4)          # everything after the raw rows is fp32 in both
    check_decay_scan("cuda", dt, 2e-5 if dt == torch.float32 else 3e-3)
    check_table_experts("cuda", dt, 2e-5 if dt == torch.float32 else 3e-2)


@pytest.mark.gpu
def test_gpu_streams_after_every_layer_run(tmp_path):
    check_streams(tmp_path, "cuda", 5e-5)


@pytest.mark.gpu
def test_gpu_long_lived_state_and_long_decoding(tmp_path):
    check_long_lived_states(tmp_path, "cuda")
    cfg = make_config(STACK, loop=LOOP)
    w = make_weights(cfg, 9)
    eng = make_engine(tmp_path, cfg, w, "float32", "cuda")
    toks = torch.randint(0, cfg["vocab"], (150,), generator=torch.Generator().manual_seed(2)).tolist()
    got = feed(eng, "x", toks, range(3, 150))
    assert rel_err(got, oracle.forward(cfg, w, toks)) < TOL["float32"]
