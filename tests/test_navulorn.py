"""Navulorn through the engine (loader, paged cache, state lines, ragged batches, scheduler) against the plain definition in
``navulorn_oracle.py``.  Every test makes its own small configuration and random checkpoint; the CPU tests run the PyTorch
definitions of the ops in float32, the ``gpu`` tests the sm_100a kernels in float32 and bfloat16."""
import json
import os

import pytest
import torch

import navulorn_oracle as oracle

PAGE = 8
LLAMA31 = dict(factor=3.0, low=1.5, high=6.0, original=60)


def attn(heads=4, kv_heads=2, dim=10, vdim=6, rot=8, base=200.0, scale=0.4, window=19, scaling=LLAMA31):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, mask=dict(size=window))
    if rot:
        m["rot"] = dict(base=base, dims=rot)
        if scaling:
            m["rot"]["scaling"] = scaling
    return m


def latent(heads=3, dim=6, rot_dim=4, vdim=10, kv_rank=14, base=90.0, scale=0.5, window=11):
    return dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, scale=scale, mask=dict(size=window), rot=dict(base=base, dims=rot_dim))


def memory(heads=3, dim=6, vdim=10, cap=5.0):
    return dict(heads=heads, dim=dim, vdim=vdim, gate_cap=cap)


def dense(ff=28):
    return dict(kind="dense", ff=ff)


def moe(experts=6, top=2, ff=14):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top))


def layer(kind, mixer, mlp):
    return dict(type=kind, mixer=mixer, mlp=mlp)


def make_config(layers, width=36, vocab=83, eps=1e-4, alpha=1.7, softcap=9.0, scale=0.7, bigram=(29, 13, 5)):
    return dict(architecture="Navulorn", layers=layers, norm=dict(eps=eps), postln_alpha=alpha, logit_softcap=softcap, vocab=vocab, width=width,
                embedding=dict(scale=scale, bigram=dict(buckets=bigram[0], mul_prev=bigram[1], mul_cur=bigram[2])))


STACK = [layer("mlstm", memory(), moe()), layer("attention", attn(), dense()), layer("latent_attention", latent(), moe(experts=5, top=3, ff=9)),
         layer("mlstm", memory(heads=2, dim=10, vdim=4, cap=8.0), None), layer("attention", attn(heads=3, kv_heads=3, dim=6, vdim=14, rot=4, window=26, scaling=None), None)]


def make_weights(cfg, seed=0):
    """Random checkpoint in the design's tensor names (bf16-representable values), every part large enough to matter."""
    g = torch.Generator().manual_seed(seed)
    r = lambda *s, std=1.0, mean=0.0: (torch.randn(s, generator=g) * std + mean).bfloat16().float()       # noqa: E731
    W, V, w = cfg["width"], cfg["vocab"], {}
    lin = lambda o, i, s=1.5: r(o, i, std=i ** -0.5 * s)       # noqa: E731
    w["embed"], w["head"], w["final.norm"] = r(V, W), lin(V, W, 3.0), r(W, std=0.3, mean=1.0)
    w["bigram"] = r(cfg["embedding"]["bigram"]["buckets"] + 1, W, std=0.6)
    for i, L in enumerate(cfg["layers"]):
        a, f, m = f"l{i}.", L["mlp"], L["mixer"]
        w[a + "norm1"] = r(W, std=0.3, mean=1.0)
        p, H, D, Dv = a + "mix.", m["heads"], m["dim"], m["vdim"]
        if L["type"] == "attention":
            G = m["kv_heads"]
            w[p + "q"], w[p + "k"], w[p + "v"], w[p + "g"] = lin(H * D, W), lin(G * D, W), lin(G * Dv, W), lin(H, W)
            w[p + "q.norm"], w[p + "k.norm"] = r(H * D, std=0.4, mean=1.2), r(G * D, std=0.4, mean=1.2)
        elif L["type"] == "latent_attention":
            R, rot = m["kv_rank"], m["rot_dim"]
            w[p + "q"], w[p + "dkv"], w[p + "dkv.norm"] = lin(H * (D + rot), W), lin(R + rot, W), r(R, std=0.3, mean=1.0)
            w[p + "uk"], w[p + "uv"] = lin(H * D, R), lin(H * Dv, R)
        else:
            w[p + "q"], w[p + "k"], w[p + "v"], w[p + "g"] = lin(H * D, W), lin(H * D, W), lin(H * Dv, W), lin(H * Dv, W)
            w[p + "i"], w[p + "f"], w[p + "i.b"], w[p + "f.b"] = lin(H, W), lin(H, W), r(H), r(H, std=0.7, mean=2.5)
            w[p + "norm"] = r(H * Dv, std=0.3, mean=1.0)
        w[p + "o"] = lin(W, H * Dv, 2.0)
        p = a + "mlp."
        if f is None:
            continue
        w[a + "norm2"] = r(W, std=0.3, mean=1.0)
        if f["kind"] == "dense":
            w[p + "gate"], w[p + "up"], w[p + "down"] = lin(f["ff"], W), lin(f["ff"], W), lin(W, f["ff"], 1.5)
        else:
            E, ff = f["router"]["experts"], f["expert"]["ff"]
            w[p + "router"], w[p + "router.b"] = lin(E, W), r(E, std=0.8)
            for e in range(E):
                w[f"{p}e{e}.gate"], w[f"{p}e{e}.up"], w[f"{p}e{e}.down"] = lin(ff, W), lin(ff, W), lin(W, ff, 1.5)
    return w


def make_engine(tmp_path, cfg, w, dtype="float32", device="cpu", max_tokens=512, max_requests=4, name="ckpt", page=PAGE):
    from safetensors.torch import save_file
    from neuronx_distributed_inference_b200.runtime.scheduler import build_engine
    d = tmp_path / name
    os.makedirs(d, exist_ok=True)
    with open(d / "config.json", "w") as f:
        json.dump(cfg, f)
    save_file({k: v.bfloat16().contiguous() for k, v in w.items()}, str(d / "model.safetensors"))
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
    """float32: the whole block within a tight relative error.  bfloat16: in stacks this narrow a router's close call or a peaked softmax
    can magnify the rounding of single positions, so positions are assessed one by one: the typical one within the tolerance, few beyond
    three times that."""
    if dtype == "float32":
        return rel_err(got, want) < TOL[dtype]
    got, want = got.double(), want.double()
    e = (got - want).norm(dim=-1) / want.norm(dim=-1).clamp_min(1e-9)
    return float(e.median()) < TOL[dtype] and float((e > 3 * TOL[dtype]).double().mean()) <= 0.1


def check_schedules(tmp_path, device, dtype, layers=STACK, T=61, seed=0, **cfg_kw):
    cfg = make_config(layers, **cfg_kw)
    w = make_weights(cfg, seed)
    eng = make_engine(tmp_path, cfg, w, dtype, device)
    toks = torch.randint(0, cfg["vocab"], (T,), generator=torch.Generator().manual_seed(seed + 1)).tolist()
    want = oracle.forward(cfg, w, toks)
    whole = feed(eng, "whole", toks, [])
    assert close(whole, want, dtype)
    eng.release("whole")
    # most of the prompt at once, the rest token by token (slot and pages of the released request are used again): memories, the carried
    # token and keys go on from where the prompt left them
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
    # one layer of each kind alone: one head, no feed-forward, a window of one or two tokens, two buckets
    ([layer("attention", attn(heads=1, kv_heads=1, dim=4, vdim=4, rot=4, window=2), None)], dict(width=20, vocab=31, bigram=(2, 1, 0))),
    ([layer("latent_attention", latent(heads=1, dim=2, rot_dim=2, vdim=3, kv_rank=4, window=1), None)], dict(width=20, vocab=31, bigram=(1, 3, 4))),
    ([layer("mlstm", memory(heads=1, dim=4, vdim=4, cap=1.0), None)], dict(width=20, vocab=31, alpha=1.0, softcap=2.0)),
    # one kv head for all heads, a rotation of two channels, values wider than keys, every expert chosen, one expert
    ([layer("attention", attn(heads=6, kv_heads=1, dim=6, vdim=20, rot=2, window=8), moe(experts=3, top=3, ff=6)),
      layer("mlstm", memory(heads=5, dim=3, vdim=20, cap=30.0), moe(experts=1, top=1))], dict(width=28, scale=1.0, alpha=0.8)),
    # sizes that coincide (width, heads, head and latent sizes), windows of a page and of two, all channels rotated, far positions scaled only
    ([layer("latent_attention", latent(heads=2, dim=8, rot_dim=8, vdim=8, kv_rank=8, window=PAGE), dense(32)),
      layer("attention", attn(heads=2, kv_heads=2, dim=8, vdim=8, rot=8, window=2 * PAGE, scaling=dict(factor=8.0, low=1.0, high=1.5, original=8)), dense(32)),
      layer("mlstm", memory(heads=2, dim=8, vdim=8), dense(32))], dict(width=32)),
    # odd sizes: width, values, latent and heads that no vector access divides; rotation by an odd number of pairs; a window past the sequence
    ([layer("mlstm", memory(heads=3, dim=7, vdim=5), moe(experts=4, top=2, ff=7)), layer("attention", attn(heads=3, kv_heads=1, dim=10, vdim=7, rot=6, window=500), dense(13)),
      layer("latent_attention", latent(heads=3, dim=5, rot_dim=2, vdim=7, kv_rank=9, window=70), None)], dict(width=35, bigram=(101, 1009, 77))),
]


@pytest.mark.parametrize("layers,kw", OTHER)
def test_other_sizes_and_layouts(tmp_path, layers, kw):
    check_schedules(tmp_path, "cpu", "float32", layers=layers, T=45, seed=5, **kw)


def test_plain_embedding_and_uncapped_logits(tmp_path):
    """A configuration without bigrams and without a logit cap."""
    cfg = make_config(STACK[:2])
    del cfg["embedding"]["bigram"]
    cfg["logit_softcap"] = None
    w = {k: v for k, v in make_weights(make_config(STACK[:2]), 1).items() if k != "bigram"}
    eng = make_engine(tmp_path, cfg, w)
    toks = list(range(5, 45))
    assert rel_err(feed(eng, 0, toks, [3, 20, 21]), oracle.forward(cfg, w, toks)) < TOL["float32"]


def _model(eng):
    return eng.app.context_encoding_model.model if hasattr(eng.app, "context_encoding_model") else eng.app.model


def check_streams(tmp_path, device, tol):
    cfg = make_config(STACK)
    w = make_weights(cfg, 2)
    eng = make_engine(tmp_path, cfg, w, device=device)
    toks = list(range(3, 20))
    streams = []
    oracle.forward(cfg, w, toks, streams)
    T = len(toks)
    on = lambda t: t.to(device)       # noqa: E731
    out = _model(eng)(on(torch.tensor([toks]).int()), attention_mask=on(torch.ones(1, T, dtype=torch.int32)), position_ids=on(torch.arange(T).view(1, T)),
                      seq_ids=on(torch.tensor([0])), slot_mapping=on(torch.arange(T).view(1, T).int()), block_table=on(torch.arange(4).view(1, 4).int()),
                      computed_context_lens=torch.tensor([0]), capture=True)
    assert len(streams) == len(STACK)
    for i, s in enumerate(streams):
        assert float((out.captured[f"layers.{i}.out"][0].double().cpu() - s).abs().max() / s.abs().max()) < tol, i


def test_streams_after_every_layer(tmp_path):
    check_streams(tmp_path, "cpu", 5e-5)


def test_long_decoding_over_many_pages(tmp_path):
    cfg = make_config(STACK)
    w = make_weights(cfg, 9)
    eng = make_engine(tmp_path, cfg, w)
    toks = torch.randint(0, cfg["vocab"], (90,), generator=torch.Generator().manual_seed(2)).tolist()
    got = feed(eng, "x", toks, range(3, 90))         # 3-token prompt, then 87 single tokens over twelve pages
    assert rel_err(got, oracle.forward(cfg, w, toks)) < TOL["float32"]


def test_cache_pool_smaller_than_all_requests(tmp_path):
    """The pool holds two requests' worth of pages: the third request runs on the pages and the slot the first gave back, and must not
    see what the first left in them (keys, memories, the carried token)."""
    cfg = make_config(STACK)
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


def check_window_reach(tmp_path, device):
    """One attention layer, one token of the prompt changed: the last position's logits move when the token lies inside its window and are
    the very same when it lies outside (the bigram table reaches one token further: the token before the window's first)."""
    for kind, mixer in (("attention", attn(window=13)), ("latent_attention", latent(window=13))):
        for hashed in (True, False):
            cfg = make_config([layer(kind, mixer, None)])
            if not hashed:
                cfg["embedding"]["bigram"] = dict(buckets=29, mul_prev=0, mul_cur=1)
            w = make_weights(cfg, 3)
            eng = make_engine(tmp_path, cfg, w, device=device, name=f"{kind}{hashed}")
            g = torch.Generator().manual_seed(4)
            for T in (26, 33, 40):                    # windows that begin inside a page, at its last and at its first token
                toks = torch.randint(1, cfg["vocab"], (T,), generator=g).tolist()
                for cuts in ([], [T - 1], [T - 2], [T - 13], [T - 14], [2, T - 5]):
                    base = feed(eng, 0, toks, cuts, want=[T - 1])
                    eng.release(0)
                    for back in (0, 1, 11, 12, 13, 14, 20, T - 1):
                        other = list(toks)
                        other[T - 1 - back] = (toks[T - 1 - back] + 5) % cfg["vocab"]
                        got = feed(eng, 0, other, cuts, want=[T - 1])
                        eng.release(0)
                        moved = rel_err(got, base)
                        assert (moved > 1e-3) if back <= 12 or (hashed and back == 13) else moved < 1e-6, (kind, hashed, T, cuts, back, moved)


def test_a_window_reaches_exactly_as_far_as_configured(tmp_path):
    check_window_reach(tmp_path, "cpu")


def check_long_lived_memory(tmp_path, device):
    """Forget gates close to one and a loud first input gate: what the first tokens wrote into the memory still shapes the logits hundreds of
    tokens on, whether the prompt arrives whole, in portions or token by token."""
    cfg = make_config([layer("mlstm", memory(cap=14.0), None), layer("mlstm", memory(heads=2, dim=8, vdim=6, cap=20.0), None)])
    w = make_weights(cfg, 1)
    for i in (0, 1):
        w[f"l{i}.mix.f.b"].fill_(9.0)
        w[f"l{i}.mix.f"] *= 0.1
        w[f"l{i}.mix.i.b"].fill_(-1.0)
    w["l0.mix.i"] *= 2
    eng = make_engine(tmp_path, cfg, w, device=device, max_tokens=1024)
    g = torch.Generator().manual_seed(8)
    toks = torch.randint(0, cfg["vocab"], (260,), generator=g).tolist()
    other = [(toks[0] + 1) % cfg["vocab"], (toks[1] + 7) % cfg["vocab"]] + toks[2:]
    want, moved = oracle.forward(cfg, w, toks), oracle.forward(cfg, w, other)
    assert rel_err(moved[-5:], want[-5:]) > 1e-3                  # the first two tokens matter at the end
    last = list(range(255, 260))
    for cuts in ([], [100, 200], [3] + list(range(230, 260))):
        got = feed(eng, "s", toks, cuts, want=last)
        eng.release("s")
        assert rel_err(got, want[-5:]) < TOL["float32"]


def test_a_long_lived_memory_carries_the_first_tokens_far(tmp_path):
    check_long_lived_memory(tmp_path, "cpu")


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


def loud_key_case(dev, dtype, target, pos, window, *, latent_rows=False, page=4, as_prompt=False, extra=0, D=8, Dv=6):
    """The key row ``target`` is made to dominate the query at ``pos`` (one query and one key are scaled so that one score stands out).
    ``latent_rows``: one row per token that is the key as a whole and the value in its first ``Dv`` numbers; otherwise four heads over two
    kv heads with a sigmoid gate per head.  Returns (op output, plain output, output when the target is all that is seen)."""
    from neuronx_distributed_inference_b200 import ops
    H, G = 4, 1 if latent_rows else 2
    g = torch.Generator().manual_seed(target * 131 + pos)
    n = pos + 1 + extra
    k, q = torch.randn(n, G, D, generator=g) * 0.1, torch.randn(n, H, D, generator=g) * 0.1
    v = torch.randn(n, G, Dv, generator=g)
    if latent_rows:
        k[..., :Dv], q[pos, :, :Dv] = v * 0.5, 0.0        # the value numbers take no part in the loud score
    loud = slice(Dv if latent_rows else 0, D)
    k[target, :, loud] = q[pos, :, loud] = (30.0 / (0.5 * (loud.stop - loud.start))) ** 0.5
    vals = k[..., :Dv] if latent_rows else v
    gate = None if latent_rows else torch.randn(n, H, generator=g)
    rd = lambda t: t.to(dtype).double()                                     # noqa: E731
    see = oracle.visible(n, dict(size=window))[:pos + 1]
    want = torch.stack([oracle.softmax_rows(rd(q[:pos + 1, h]) @ rd(k[:, h // (H // G)]).T * 0.5, see) @ rd(vals[:, h // (H // G)]) for h in range(H)], 1)[pos]
    sg = torch.ones(H) if gate is None else torch.sigmoid(gate[pos])
    kc, table = paged(k, page, torch.Generator().manual_seed(5))
    vc = kc if latent_rows else paged(v, page, torch.Generator().manual_seed(5))[0]
    to = lambda t: None if t is None else t.to(dev, dtype)                                      # noqa: E731
    kc = to(kc)
    vc = kc if latent_rows else to(vc)
    kw = dict(value_dim=Dv) if latent_rows else dict(gate_per_head=True)
    if as_prompt:
        got = ops.paged_window_attention(to(q.view(1, n, H, D)), kc, vc, table.to(dev), i32(dev, 0), i32(dev, n), 0.5, None, window, 0,
                                         to(None if gate is None else gate.view(1, n, H)), **kw)[0, pos]
    else:
        got = ops.paged_window_attention(to(q[pos].view(1, 1, H, D)), kc, vc, table.to(dev), i32(dev, pos), i32(dev, 1), 0.5, None, window, 0,
                                         to(None if gate is None else gate[pos].view(1, 1, H)), **kw)
    row = vals[target].repeat_interleave(H // G, 0) * sg.view(H, 1)
    return got.float().cpu().view(H, Dv), (want * sg.double().view(H, 1)).float(), row


# (position, distance of the loud key, window): far keys, page borders (pages of 4), the first tokens, both sides of the window's edge
PLACES = [(300, 250, 300), (301, 40, 64), (300, 63, 64), (300, 64, 64), (64, 63, 64), (64, 64, 64), (63, 63, 64), (0, 0, 5), (4, 4, 5), (5, 5, 5), (8, 1, 9), (40, 2, 3), (40, 3, 3),
          (41, 0, 1), (41, 1, 1), (130, 89, 90), (130, 90, 90)]


@pytest.mark.parametrize("pos,back,window", PLACES)
@pytest.mark.parametrize("as_prompt", [False, True])
@pytest.mark.parametrize("latent_rows", [False, True])
def test_loud_keys_near_and_far_and_at_the_windows_edge(pos, back, window, as_prompt, latent_rows):
    got, want, row = loud_key_case("cpu", torch.float32, pos - back, pos, window, as_prompt=as_prompt, latent_rows=latent_rows, D=10 if latent_rows else 8)
    assert torch.allclose(got, want, atol=1e-4)
    assert torch.allclose(got, row, atol=2e-2) == (back < window)


def test_a_prompt_does_not_see_later_rows_of_its_portion():
    for lat in (False, True):
        got, want, row = loud_key_case("cpu", torch.float32, 21, 20, 12, as_prompt=True, extra=3, latent_rows=lat, D=10 if lat else 8)       # the loud row is one step ahead
        assert torch.allclose(got, want, atol=1e-4) and not torch.allclose(got, row, atol=0.2)


def unequal_portions(T, sizes, run, B=2):
    """Feed ``B`` rows of ``T`` tokens in unequal portions through ``run(at, n)`` -> [B, max(n), C]; the rows put together again."""
    at, rows, step = [0] * B, [[] for _ in range(B)], 0
    while min(at) < T:
        n = [min(T - at[b], sizes[(step + b) % len(sizes)]) for b in range(B)]
        y = run(at, n)
        for b in range(B):
            rows[b].append(y[b, :n[b]].double().cpu())
            at[b] += n[b]
        step += 1
    return [torch.cat(r) for r in rows]


def cut(x, at, n):
    out = torch.zeros(x.shape[0], max(n), *x.shape[2:], dtype=x.dtype)
    for b in range(x.shape[0]):
        out[b, :n[b]] = x[b, at[b]:at[b] + n[b]]
    return out


def check_bigrams(dev, dt, tol):
    """Rows of the bigram table and the carried token: whole rows, unequal portions, lines that hold another request's token, row lengths
    of zero, products beyond 32 bits, a scale of one, no table at all."""
    from neuronx_distributed_inference_b200 import ops
    g = torch.Generator().manual_seed(0)
    for W, V, b in ((36, 50, (29, 13, 5)), (35, 400, (1, 3, 4)), (256, 1000, (977, 3000017, 70001)), (1024, 60, (2, 1, 0))):
        B, T = 2, 23
        e, t2 = (torch.randn(V, W, generator=g)).to(dt), torch.randn(b[0] + 1, W, generator=g).to(dt)
        ids = torch.randint(0, V, (B, T), generator=g).int()
        spec = dict(buckets=b[0], mul_prev=b[1], mul_cur=b[2])
        w = dict(embed=e.double(), bigram=t2.double())
        want = [oracle.embedding(ids[r].tolist(), w, dict(scale=0.6, bigram=spec)) for r in range(B)]
        st = torch.full((5, 1), 7, dtype=torch.int32).to(dev)
        args = (e.to(dev), t2.to(dev), 0.6, b[1], b[2], st)
        x, lp = ops.bigram_embed(ids.to(dev), *args, i32(dev, 3, 1), i32(dev, 0, 0), i32(dev, T, T - 4), torch.bfloat16)
        assert torch.allclose(x[0].double().cpu(), want[0], atol=1e-6) and torch.allclose(x[1, :T - 4].double().cpu(), want[1][:T - 4], atol=1e-6)
        assert not x[1, T - 4:].any() and torch.equal(lp, x.bfloat16())
        assert st.view(-1).tolist() == [7, int(ids[1, T - 5]), 7, int(ids[0, -1]), 7]
        got = unequal_portions(T, [1, 2, 6], lambda at, n: ops.bigram_embed(cut(ids, at, n).to(dev), *args, i32(dev, 0, 4), i32(dev, *at), i32(dev, *n))[0])
        assert all(torch.allclose(got[r], want[r], atol=1e-6) for r in range(B))
        x, lp = ops.bigram_embed(ids.to(dev), e.to(dev), None, 1.0, 0, 0, None, i32(dev, 3, 1), i32(dev, 0, 0), i32(dev, T, 0))
        assert lp is None and torch.equal(x[0].cpu(), e[ids[0].long()].float()) and not x[1].any()


def rope_cos_sin(rot, ctx, T, dev):
    ang = (ctx.double().view(-1, 1) + torch.arange(T).double().view(1, T)).unsqueeze(-1) * oracle.frequencies(rot)
    return torch.cos(ang).float().to(dev), torch.sin(ang).float().to(dev)


def rotated(rows, rot, at, interleaved):
    """The oracle's rotation of rows that stand at positions ``at`` .. of a sequence."""
    pad = torch.zeros(at, *rows.shape[1:], dtype=rows.dtype)
    return oracle.rotate(torch.cat([pad, rows]), rot, interleaved)[at:]


def check_norm_rope_append(dev, dt, tol):
    """Row-wide q / k norms, both rotation layouts (odd numbers of pairs too) and the cache rows, without a convolution, behind a context."""
    from neuronx_distributed_inference_b200 import ops
    g = torch.Generator().manual_seed(1)
    rn = lambda *s: torch.randn(*s, generator=g)        # noqa: E731
    B, T, page, nblk, eps = 3, 11, 4, 14, 1e-3
    ctx, ql = torch.tensor([0, 5, 40]).int(), torch.tensor([T, 4, 1]).int()
    for H, G, D, Dv, R in ((4, 2, 10, 6, 8), (3, 1, 10, 7, 6), (2, 2, 16, 16, 0), (4, 2, 64, 128, 64), (2, 1, 12, 8, 2), (5, 1, 24, 16, 16), (6, 3, 128, 64, 96),
                         (3, 3, 32, 8, 8)):
        C = H * D + G * (D + Dv)
        p = rn(B, T, -(-(C + H) // 8) * 8).to(dt)
        qw, kw = rn(H * D) * 0.3 + 1, rn(G * D) * 0.3 + 1
        rot = dict(base=77.0, dims=R, scaling=LLAMA31)
        cos, sin = rope_cos_sin(rot, ctx, T, dev) if R else (None, None)
        table = torch.randperm(B * nblk, generator=g).view(B, nblk).int()
        for half in (True, False):
            kd, vd = torch.zeros(B * nblk, page, G, D, dtype=dt).to(dev), torch.zeros(B * nblk, page, G, Dv, dtype=dt).to(dev)
            q = ops.conv_qknorm_rope_append(p.to(dev), None, None, i32(dev, 0, 1, 2), ctx.to(dev), ql.to(dev), qw.to(dev), kw.to(dev), eps, H, G, D, Dv,
                                            cos, sin, kd, vd, table.to(dev), half=half)
            for b in range(B):
                n, c0 = int(ql[b]), int(ctx[b])
                rows = p[b, :n].double()
                turn = (lambda x: rotated(x, rot, c0, not half)) if R else (lambda x: x)
                qd = turn((oracle.rms(rows[:, :H * D], eps) * qw.double()).view(n, H, D))
                kk = turn((oracle.rms(rows[:, H * D:(H + G) * D], eps) * kw.double()).view(n, G, D))
                assert torch.allclose(q[b, :n].double().cpu(), qd, atol=tol * 3, rtol=tol)
                for t in range(n):
                    at = (int(table[b, (c0 + t) // page]), (c0 + t) % page)
                    assert torch.allclose(kd[at].double().cpu(), kk[t], atol=tol * 3, rtol=tol)
                    assert torch.equal(vd[at].double().cpu(), rows[t, (H + G) * D:C].view(G, Dv))


def check_latent_rows(dev, dt, tol):
    """Latent norm, rotated shared key part and rotated query channels in both layouts."""
    from neuronx_distributed_inference_b200 import ops
    g = torch.Generator().manual_seed(2)
    rn = lambda *s: torch.randn(*s, generator=g)        # noqa: E731
    B, T, page, nblk, eps = 3, 9, 4, 14, 1e-3
    ctx, ql = torch.tensor([0, 5, 40]).int(), torch.tensor([T, 4, 1]).int()
    for H, D, R, rot_dim in ((3, 6, 14, 4), (2, 5, 9, 2), (4, 40, 88, 24), (1, 2, 300, 10)):
        p = rn(B, T, H * (D + rot_dim) + R + rot_dim).to(dt)
        wn = rn(R) * 0.3 + 1
        rot = dict(base=55.0, dims=rot_dim)
        cos, sin = rope_cos_sin(rot, ctx, T, dev)
        table = torch.randperm(B * nblk, generator=g).view(B, nblk).int()
        for inter in (True, False):
            cache = torch.zeros(B * nblk, page, 1, R + rot_dim, dtype=dt).to(dev)
            off = H * (D + rot_dim)
            ops.latent_norm_append(p.to(dev), off, R, wn.to(dev), eps, cache, table.to(dev), ctx.to(dev), ql.to(dev), rot_dim=rot_dim, cos=cos, sin=sin, interleaved=inter)
            a = torch.zeros(B, T, H, R + rot_dim, dtype=dt).to(dev)
            ops.rope_tail(p[..., :off].reshape(B, T, H, D + rot_dim).contiguous().to(dev), a, rot_dim, cos, sin, inter)
            for b in range(B):
                n, c0 = int(ql[b]), int(ctx[b])
                rows = p[b, :n].double()
                c = oracle.rms(rows[:, off:off + R], eps) * wn.double()
                kr = rotated(rows[:, off + R:], rot, c0, inter)
                qr = rotated(rows[:, :off].view(n, H, D + rot_dim)[..., D:], rot, c0, inter)
                assert torch.allclose(a[b, :n, :, R:].double().cpu(), qr, atol=tol * 3, rtol=tol)
                for t in range(n):
                    at = (int(table[b, (c0 + t) // page]), (c0 + t) % page)
                    assert torch.allclose(cache[at][0].double().cpu(), torch.cat([c[t], kr[t]]), atol=tol * 3, rtol=tol)


MEMORY_SIZES = ((3, 6, 10, 37), (2, 7, 5, 18), (4, 64, 64, 150), (2, 128, 40, 200), (2, 64, 16, 65), (1, 136, 20, 35), (2, 40, 56, 70), (1, 256, 24, 90), (3, 20, 100, 64))


def check_memory(dev, dt, tol, sizes=MEMORY_SIZES, spread=1.0, f_mean=2.0):
    """Matrix memory against the plain loop: whole rows and unequal portions with carried memory, key sum and maximum; lines that hold
    another request's state; gates that reach their cap; then the per-head norm with a weight per channel and the sigmoid gate."""
    from neuronx_distributed_inference_b200 import ops
    g = torch.Generator().manual_seed(3)
    rn = lambda *s: torch.randn(*s, generator=g)        # noqa: E731
    on = lambda t: t.to(dev)      # noqa: E731
    for H, D, Dv, T in sizes:
        B, cap, NS = 2, 6.0, -(-Dv // ops.MLSTM_SLICE)
        C = H * (2 * D + Dv)
        at_g = C + H * Dv
        p = torch.cat([rn(B, T, at_g), rn(B, T, 2 * H) * 2 * spread, torch.zeros(B, T, -(at_g + 2 * H) % 8)], -1).to(dt)
        ib, fb = rn(H) * spread, rn(H) + f_mean
        raw = p[..., at_g:at_g + 2 * H].double()
        soft = lambda z: cap * torch.tanh(z / cap)      # noqa: E731
        gi, gf = soft(raw[..., :H] + ib.double()), torch.nn.functional.logsigmoid(soft(raw[..., H:] + fb.double()))
        q, k, v = (t.double().reshape(B, T, H, -1) for t in p[..., :C].split([H * D, H * D, H * Dv], -1))
        want = torch.stack([oracle.mlstm_states(q[b] * D ** -0.5, k[b], v[b], gi[b], gf[b]) for b in range(B)]).reshape(B, T, -1)
        # where the denominator nearly vanishes before its floor the quotient magnifies any rounding: assess relative to the row's size
        size = want.reshape(B, T, H, Dv).norm(dim=-1, keepdim=True).expand(-1, -1, -1, Dv).reshape(want.shape) + 0.05
        fresh = lambda: (on(rn(5, H, Dv, D) * 9), on(rn(5, H, NS, D) * 9), on(rn(5, H, NS) * 9))       # noqa: E731  (left by earlier requests)
        st = fresh()
        args = (at_g, on(ib), on(fb), cap)
        y = ops.mlstm_scan(on(p), *args, *st, i32(dev, 3, 1), i32(dev, 0, 0), i32(dev, T, T), H, D, Dv)
        assert float(((y.double().cpu() - want).abs() / size).max()) < tol, (H, D, Dv, T)
        st2 = fresh()
        got = unequal_portions(T, [1, 2, 19, 70], lambda at, n: ops.mlstm_scan(on(cut(p, at, n)), *args, *st2, i32(dev, 0, 4), i32(dev, *at), i32(dev, *n), H, D, Dv))
        for b in range(B):
            assert float(((got[b] - want[b]).abs() / size[b]).max()) < tol, (H, D, Dv, T)
        for x, z in zip(st, st2):
            big = float(x[[1, 3]].abs().max())
            assert torch.allclose(z[0], x[3], atol=tol * big, rtol=tol) and torch.allclose(z[4], x[1], atol=tol * big, rtol=tol)
        for x in st[1:]:        # every copy of the key sum and of the maximum is the same
            assert torch.equal(x[3], x[3][:, :1].expand_as(x[3]))
        wn = rn(H * Dv)
        gate = on(p)[..., C:at_g]
        o = ops.head_rmsnorm_gate(y, on(wn), H, 1e-3, gate, "sigmoid", out_dtype=dt)
        o_want = oracle.rms(y.double().cpu().view(B, T, H, Dv), 1e-3).reshape(B, T, -1) * wn.double() * torch.sigmoid(p[..., C:at_g].double())
        otol = 1e-2 if dt == torch.bfloat16 else 2e-5
        assert torch.allclose(o.double().cpu(), o_want, atol=otol, rtol=otol)


def check_router(dev, dt):
    """Biased router, softmax over the chosen logits: the bias decides who is chosen and counts in the weights."""
    from neuronx_distributed_inference_b200.modules.moe import RouterTopK
    g = torch.Generator().manual_seed(4)
    for W, E, k, N in ((36, 6, 2, 5), (64, 12, 3, 100), (35, 5, 5, 3), (128, 1, 1, 9), (336, 64, 6, 70)):
        r = RouterTopK(E, k, W, dt, "softmax", True, True, True, dev)
        wt, b = torch.randn(E, W, generator=g) * W ** -0.5, torch.randn(E, generator=g) * 3
        b[0] += 60.0          # far ahead: the others' scores vanish in a softmax over all, not in the choice
        r.linear_router.weight.copy_(wt)
        r.linear_router.bias.copy_(b)
        x = torch.randn(N, W, generator=g).to(dt)
        logits, w, idx = r(x.to(dev))
        z = x.double() @ wt.double().T + b.double()
        ww, wi = oracle.route(z, k)
        assert torch.allclose(logits.double().cpu(), z, atol=1e-4)
        assert torch.equal(idx.long().cpu(), wi) and torch.allclose(w.double().cpu(), ww, atol=1e-5)


def check_dense_and_sum_norm(dev, dt, tol):
    from neuronx_distributed_inference_b200 import ops
    g = torch.Generator().manual_seed(5)
    rn = lambda *s: torch.randn(*s, generator=g)        # noqa: E731
    for W, ff, N in ((36, 28, 5), (64, 128, 40), (35, 13, 9), (256, 192, 3)):
        x, gu = rn(N, W).to(dt), (rn(2 * ff, W) * W ** -0.5 * 2).to(dt)
        y = ops.linear(x.to(dev).view(1, N, W), gu.to(dev), act="gelu_tanh_mul").view(N, ff)
        z = x.double() @ gu.double().T
        assert torch.allclose(y.double().cpu(), oracle.gelu_tanh(z[:, :ff]) * z[:, ff:], atol=tol * 6, rtol=tol)
    for W in (36, 35, 256, 1028, 5120, 9000):
        x, y, wn = rn(7, W), rn(7, W).to(dt), rn(W)
        out, lp = ops.scaled_add_rmsnorm(x.to(dev), y.to(dev), wn.to(dev), 1.7, 1e-3, 0.0, torch.bfloat16)
        want = oracle.rms(1.7 * x.double() + y.double(), 1e-3) * wn.double()
        assert torch.allclose(out.double().cpu(), want, atol=2e-5, rtol=2e-5) and torch.equal(lp, out.bfloat16())
        out, _ = ops.scaled_add_rmsnorm(x.to(dev), None, wn.to(dev), 0.5, 1e-3, 1.0)
        assert torch.allclose(out.double().cpu(), oracle.rms(0.5 * x.double(), 1e-3) * (1 + wn.double()), atol=2e-5, rtol=2e-5)


def test_bigram_rows_and_the_carried_token():
    check_bigrams("cpu", torch.float32, 1e-6)


def test_row_norms_rotation_layouts_and_cache_rows():
    check_norm_rope_append("cpu", torch.float32, 1e-5)


def test_latent_rows_and_rotated_query_channels():
    check_latent_rows("cpu", torch.float32, 1e-5)


def test_matrix_memory_and_what_it_carries():
    check_memory("cpu", torch.float32, 1e-3)
    check_memory("cpu", torch.float32, 1e-3, MEMORY_SIZES[:2], spread=6.0, f_mean=-1.0)          # gates at their caps, memories that fade at once


def test_biased_router_and_softmax_over_the_chosen():
    check_router("cpu", torch.float32)


def test_gelu_gate_product_and_post_norm():
    check_dense_and_sum_norm("cpu", torch.float32, 1e-5)


def test_frequencies_follow_the_wavelength():
    """Short wavelengths keep their frequency, long ones are divided by the factor, a blend in between; borders of every kind occur."""
    from neuronx_distributed_inference_b200.models.navulorn.modeling_navulorn import rope_of
    for sc in (LLAMA31, dict(factor=8.0, low=1.0, high=4.0, original=512), None):
        rot = dict(dims=20, base=3000.0)
        if sc:
            rot["scaling"] = sc
        inv, mag, _ = rope_of(rot)
        want = oracle.frequencies(rot)
        assert mag == 1.0 and torch.allclose(inv, want, rtol=1e-12)
        if sc:
            ratio = want / oracle.frequencies(dict(dims=20, base=3000.0))
            kinds = {"kept" if r > 1 - 1e-9 else "slow" if r < 1 / sc["factor"] + 1e-9 else "blend" for r in ratio.tolist()}
            assert kinds == {"kept", "slow", "blend"}


def test_registry_picks_the_model_from_config_json(tmp_path):
    from neuronx_distributed_inference_b200.utils.constants import get_model_cls, model_type_of
    with open(tmp_path / "config.json", "w") as f:
        json.dump(make_config(STACK), f)
    assert get_model_cls(model_type_of(str(tmp_path))).__name__ == "NeuronNavulornForCausalLM"


def test_unknown_parts_are_refused(tmp_path):
    for i, bad in enumerate(([layer("rwkv", memory(), None)], [layer("mlstm", memory(), dict(kind="other"))],
                             [layer("latent_attention", dict(latent(), rot=dict(base=9.0, dims=2)), None)])):
        cfg = make_config(bad)
        with pytest.raises(ValueError):
            make_engine(tmp_path, cfg, {"embed": torch.zeros(1)}, name=f"bad{i}")


def test_command_line_generates_from_token_ids(tmp_path, capsys):
    from neuronx_distributed_inference_b200 import inference_demo
    cfg = make_config(STACK)
    w = make_weights(cfg)
    eng = make_engine(tmp_path, cfg, w)
    want = eng.generate([[1, 2, 3, 4], [7, 8]], 5)
    inference_demo.main(["--model-type", "navulorn", "--task-type", "causal-lm", "run", "--model-path", str(tmp_path / "ckpt"),
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
    for k in ("bigram_embed", "scaled_add_rmsnorm", "conv_qknorm_rope_append", "paged_window_attention", "latent_norm_append", "rope_tail", "mlstm_scan",
              "head_rmsnorm_gate", "router_topk", "gated_act_mul", "moe_plain_gated"):
        assert ops.stats[k] > 0, k
    tkg = eng.app.token_generation_model          # single-token steps replayed from CUDA graphs (capture did not fall back to eager)
    assert tkg.use_graphs and len(tkg._graphs) > 0


# head sizes of 64 and 128 (tensor-core attention and chunked memories on bf16 portions, grouped expert GEMMs) beside sizes that take the
# CUDA-core kernels; memories with 128 and 136 key channels.  Stacks of two or three layers: a deeper one of random routers magnifies bf16
# rounding until nothing can be said about single positions
WIDER = [
    [layer("attention", attn(heads=4, kv_heads=2, dim=64, vdim=128, rot=32, scale=0.12, window=40), moe(experts=6, top=2, ff=128)),
     layer("mlstm", memory(heads=4, dim=64, vdim=48, cap=9.0), dense(256))],
    [layer("latent_attention", latent(heads=4, dim=32, rot_dim=64, vdim=64, kv_rank=128, scale=0.1, window=37), moe(experts=8, top=3, ff=64)),
     layer("mlstm", memory(heads=2, dim=128, vdim=64), dense(96))],
    [layer("attention", attn(heads=2, kv_heads=1, dim=128, vdim=64, rot=128, scale=0.09, window=64), dense(192)), layer("mlstm", memory(heads=1, dim=136, vdim=20), None),
     layer("latent_attention", latent(heads=2, dim=16, rot_dim=16, vdim=24, kv_rank=64, scale=0.2, window=30), moe(experts=5, top=1, ff=96))],
    [layer("attention", attn(heads=8, kv_heads=2, dim=80, vdim=96, rot=40, scale=0.11, window=50), dense(160)),
     layer("latent_attention", latent(heads=4, dim=48, rot_dim=24, vdim=40, kv_rank=104, scale=0.1, window=33), None)],
    [layer("latent_attention", latent(heads=2, dim=16, rot_dim=32, vdim=24, kv_rank=320, scale=0.15, window=70), dense(128)),
     layer("mlstm", memory(heads=1, dim=64, vdim=272), None)],
]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("layers", WIDER)
def test_gpu_wider_stacks(tmp_path, dtype, layers):
    eng, cfg, w = check_schedules(tmp_path, "cuda", dtype, layers=layers, T=150, width=256, vocab=301, eps=1e-6, seed=7, alpha=2.0)
    check_mixed_batches(eng, cfg, w, dtype, n_req=5)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("layers,kw", OTHER)
def test_gpu_other_sizes_and_layouts(tmp_path, dtype, layers, kw):
    check_schedules(tmp_path, "cuda", dtype, layers=layers, T=45, seed=5, **kw)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("as_prompt", [False, True])
@pytest.mark.parametrize("latent_rows,D,Dv", [(False, 8, 6), (False, 64, 128), (False, 128, 64), (False, 40, 72), (True, 10, 6), (True, 80, 64), (True, 112, 88),
                                              (True, 410, 400)])
def test_gpu_loud_keys_near_and_far_and_at_the_windows_edge(dtype, as_prompt, latent_rows, D, Dv):
    for pos, back, window in PLACES:
        got, want, row = loud_key_case("cuda", dtype, pos - back, pos, window, as_prompt=as_prompt, latent_rows=latent_rows, D=D, Dv=Dv)
        assert torch.allclose(got, want, atol=2e-4 if dtype == torch.float32 else 4e-2), (pos, back, window)
        assert torch.allclose(got, row, atol=6e-2) == (back < window), (pos, back, window)


@pytest.mark.gpu
@pytest.mark.parametrize("dt,tol", [(torch.float32, 2e-5), (torch.bfloat16, 1e-2)])
def test_gpu_kernels_match_the_plain_functions(dt, tol):
    check_bigrams("cuda", dt, tol)
    check_norm_rope_append("cuda", dt, tol)
    check_latent_rows("cuda", dt, tol)
    check_memory("cuda", dt, 2e-3 if dt == torch.float32 else 6e-3)          # everything after the raw rows is fp32 (or pairs of bf16) in both
    check_memory("cuda", dt, 2e-3 if dt == torch.float32 else 6e-3, MEMORY_SIZES[:5], spread=6.0, f_mean=-1.0)
    check_memory("cuda", dt, 2e-3 if dt == torch.float32 else 6e-3, MEMORY_SIZES[2:5], spread=0.5, f_mean=8.0)
    check_router("cuda", dt)
    check_dense_and_sum_norm("cuda", dt, tol)


@pytest.mark.gpu
def test_gpu_streams_after_every_layer(tmp_path):
    check_streams(tmp_path, "cuda", 5e-5)


@pytest.mark.gpu
def test_gpu_window_reach_long_lived_memory_and_long_decoding(tmp_path):
    check_window_reach(tmp_path, "cuda")
    check_long_lived_memory(tmp_path, "cuda")
    cfg = make_config(STACK)
    w = make_weights(cfg, 9)
    eng = make_engine(tmp_path, cfg, w, "float32", "cuda")
    toks = torch.randint(0, cfg["vocab"], (150,), generator=torch.Generator().manual_seed(2)).tolist()
    got = feed(eng, "x", toks, range(3, 150))
    assert rel_err(got, oracle.forward(cfg, w, toks)) < TOL["float32"]
