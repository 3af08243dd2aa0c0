"""Nibelix on the GPU against the plain float64 oracle (oracle/nibelix_oracle.py): every mechanism's kernel
alone, then whole models (own small configurations, random weights) under every way the engine can be driven:
whole prompts, token-by-token decoding, portions down to two tokens, mixed batches of unequal requests, pages
and slots that are freed and reused, long decoding, greedy generation through the scheduler, the command line
and the trace runner."""
import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch

from oracle import nibelix_oracle as O

pytestmark = pytest.mark.gpu
BF, F32, F64 = torch.bfloat16, torch.float32, torch.float64
ROOT = Path(__file__).resolve().parent.parent


def _ops():
    from vila_b200 import ops
    return ops


def rel(a, b):
    a, b = a.double().cpu(), b.double().cpu()
    return float((a - b).abs().max() / b.abs().max().clamp_min(1e-30))


def tol(dtype):
    return 2e-5 if dtype == F32 else 5e-2   # max abs error over the largest expected entry


def rnd(*shape, seed=0, scale=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=F64) * scale


def dev(t, dtype=F32):
    return t.to(device="cuda", dtype=dtype).contiguous()


def i32(rows):
    return torch.tensor(rows, dtype=torch.int32, device="cuda")


def f32(t):
    return t.float().double()


# ------------------------------------------------------------------------------------------------
# configurations (none of them a size combination of a published or given model)
# ------------------------------------------------------------------------------------------------
def lightning(dim, vdim, decay):
    return "lightning", {"decay": list(decay), "dim": dim, "heads": len(decay), "vdim": vdim}


def attention(heads, kv_heads, dim, vdim, rot, window, *, base=10000.0, diff=0.3, scale=None):
    return "attention", {"diff": diff, "dim": dim, "heads": heads, "kv_heads": kv_heads, "mask": {"size": window},
                         "rot": {"base": base, "dims": rot}, "scale": scale if scale is not None else dim ** -0.5, "vdim": vdim}


def dense(ff):
    return {"ff": ff, "kind": "dense"}


def moe(experts, identity, top, ff, count=1, keep=1, scale=1.0, shared=0):
    m = {"expert": {"ff": ff}, "kind": "moe", "router": {"experts": experts, "groups": {"count": count, "keep": keep},
                                                          "identity": identity, "scale": scale, "top": top}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def config(width, vocab, layers, *, eps=1e-5, mult=0.5, cap=20.0):
    return {"architecture": "Nibelix", "layers": [{"mixer": m, "mlp": f, "type": t} for (t, m), f in layers],
            "logit_softcap": cap, "norm": {"eps": eps}, "residual_mult": mult, "vocab": vocab, "width": width}


CONFIGS = {
    # nothing is a multiple of 8: every projection runs on the CUDA-core kernel in both dtypes; an attention layer first, a
    # window that is shorter than a key block and one that crosses pages; a layer without feed-forward; all three router forms
    "odd": config(92, 113, [
        (attention(6, 2, 10, 14, 6, 37, base=500.0, diff=0.7), moe(9, 3, 4, 20, count=4, keep=2, scale=2.5, shared=28)),
        (lightning(7, 9, [0.3, 0.99, 0.9]), dense(36)),
        (attention(3, 3, 9, 5, 4, 90, scale=0.6), None),
        (lightning(12, 20, [0.97, 0.5]), moe(5, 1, 3, 12, count=3, keep=3)),
        (attention(4, 1, 12, 22, 12, 5, diff=0.2), moe(6, 0, 1, 16, count=2, keep=1, scale=0.7, shared=4))], mult=0.4),
    # tensor-core shapes; dense and routed feed-forwards on both mixers; one key head for 8 query heads
    "aligned": config(128, 256, [
        (lightning(32, 48, [0.6, 0.8, 0.95, 0.999]), dense(64)),
        (attention(8, 1, 32, 40, 8, 64, base=1e6), dense(160)),
        (attention(8, 4, 16, 32, 16, 100), moe(14, 2, 4, 64, count=4, keep=2, scale=1.7, shared=96)),
        (lightning(64, 16, [0.9] * 8), moe(8, 8, 3, 32, count=2, keep=1, scale=3.0))], eps=1e-6, mult=1.0, cap=5.0),
    # values that other models make larger: one head, one expert, one choice, a window of two and of one token; no cap, no
    # decay at all, no rotation, a feed-forward of one unit, a state of 130 key channels
    "ones": config(64, 97, [
        (lightning(130, 11, [1.0]), moe(1, 0, 1, 8, scale=0.5)),
        (attention(1, 1, 8, 16, 2, 2), dense(1)),
        (lightning(9, 24, [0.0]), moe(1, 1, 2, 24, shared=1)),
        (attention(2, 2, 24, 8, 24, 1, diff=0.9), None),
        (attention(2, 1, 6, 12, 0, 700), dense(16))], mult=0.8, cap=0.0),
    # heads wider than tall and taller than wide; only recurrent layers: no paged pool at all
    "recurrent": config(72, 80, [
        (lightning(20, 66, [0.9, 0.8, 0.7, 0.6, 0.5]), dense(24)),
        (lightning(36, 8, [0.999] * 10), moe(12, 4, 5, 10, count=8, keep=4, scale=1.2, shared=20))]),
}


def build(name, dtype, seed=0):
    """name: a key of CONFIGS or a configuration"""
    from vila_b200.model import NibelixConfig, NibelixForCausalLM
    cfg = CONFIGS[name] if isinstance(name, str) else name
    model = NibelixForCausalLM(NibelixConfig.from_dict(cfg), "cuda", dtype).init_random(seed, scale=1.5)
    if dtype == BF:
        # Two choice scores closer than the bf16 noise of the router's input would pick another expert than the float64
        # oracle, and the changed token would then be seen by every later one: the bf16 models get corrections 2 apart, so
        # that the chosen set is fixed per layer while the weights still vary per token.  Routing that changes from token to
        # token is covered by the fp32 models and the router's own test.
        t = model.state_dict()
        g = torch.Generator().manual_seed(seed + 100)
        for n in t:
            if n.endswith("correction"):
                t[n] = (2.0 * torch.randperm(t[n].numel(), generator=g).float() - t[n].numel()).to(BF)
        model.load_weights(t)
    return cfg, model


def tokens_for(cfg, n, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()


def run_schedule(model, prompts, schedule, max_tokens, slots=4):
    """schedule: steps of [(name, rows)]; the logits of every row are collected per request; a request
    is released with its last row.  -> {name: [len, vocab] fp32 on the CPU}"""
    from vila_b200.serving import TokenEngine
    eng = TokenEngine(model, max_tokens=max_tokens, slots=slots)
    at = {k: 0 for k in prompts}
    got = {k: [] for k in prompts}
    for step in schedule:
        entries = []
        for name, n in step:
            entries.append((name, prompts[name][at[name]:at[name] + n], list(range(n))))
            at[name] += n
        lg = eng.step(entries).cpu()
        o = 0
        for name, n in step:
            got[name].append(lg[o:o + n])
            o += n
            if at[name] == len(prompts[name]):
                eng.release(name)
    assert not eng.seqs and eng.cache.allocator.available == eng.cache.n_pages
    return {k: torch.cat(v) for k, v in got.items()}


def rows_close(got, want, dtype, what="", per=50):
    """every row within tolerance (relative to the largest entry of the expected tensor).  bfloat16: read-outs and combined
    maps are divided by their own root mean square, so a row that nearly cancels has the bf16 noise of the projections
    multiplied; one row in `per` may leave the tolerance, none by more than 8 times.  float32: no exception."""
    got, want = got.double().cpu(), want.double().cpu()
    assert bool(torch.isfinite(got).all()), what
    err = (got - want).abs().amax(-1) / want.abs().max()
    bad = int((err >= tol(dtype)).sum())
    allowed = 0 if dtype == F32 else max(1, err.numel() // per)
    assert bad <= allowed and float(err.max()) < (1 if dtype == F32 else 8) * tol(dtype), (what, bad, err.numel(), float(err.max()))


def rare(cfg):
    return 8 if any(spec["mixer"]["heads"] == 1 for spec in cfg["layers"]) else 50


def check_logits(cfg, model, prompts, got, dtype):
    for name, toks in prompts.items():
        want = O.forward(cfg, model.state_dict(), toks)
        assert got[name].shape == want.shape
        rows_close(got[name], want, dtype, name, rare(cfg))


# ------------------------------------------------------------------------------------------------
# mechanisms alone: the recurrence
# ------------------------------------------------------------------------------------------------
def decay_inputs(T, H, d, dv, dtype, seed=0):
    r = {n: rnd(T, H, s, seed=seed + i).to(dtype) for i, (n, s) in enumerate((("q", d), ("k", d), ("v", dv)))}
    r["decay"] = torch.rand(H, generator=torch.Generator().manual_seed(seed + 9)) * 0.6 + 0.4
    return r


def decay_expected(r, q_scale, silu):
    """-> read-outs [T, H, dv], final states [H, dv, d]"""
    act = O.silu if silu else (lambda u: u)
    q, k, v = (act(r[n].double()) for n in "qkv")
    out = [O.lightning_rule(q[:, h] * q_scale, k[:, h], v[:, h], float(r["decay"][h])) for h in range(q.shape[1])]
    return torch.stack([o for o, _ in out], 1), torch.stack([S.T for _, S in out])


def run_decay(r, rows, dtype, state, seqs, q_scale, silu):
    """q | v | k side by side with a gap"""
    T, H, d = r["q"].shape
    dv = r["v"].shape[2]
    wide = torch.cat([r["q"].reshape(T, -1), torch.zeros(T, 1, dtype=dtype), r["v"].reshape(T, -1), r["k"].reshape(T, -1)], 1)
    wide = dev(wide[rows], dtype)
    vo = H * d + 1
    return _ops().decay_scan(wide[:, :H * d], wide[:, vo + H * dv:], wide[:, vo:vo + H * dv], state, seqs, heads=H, dim=d, vdim=dv,
                             decay=dev(r["decay"]), silu=silu, q_scale=q_scale)


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("H,d,dv,silu", [(3, 7, 9, True), (4, 32, 48, True), (2, 128, 64, False), (1, 130, 1, True), (2, 260, 7, False),
                                         (5, 1, 66, True), (64, 12, 320, True), (6, 64, 128, True)])
def test_decay_scan_in_portions_through_stale_slots(cuda, dtype, H, d, dv, silu):
    T, qs = (40, 0.3) if H == 64 else (70, 1.0)
    r = decay_inputs(T, H, d, dv, dtype)
    want, S = decay_expected(r, qs, silu)
    state = torch.full((3, H, dv, d), -9.0, device="cuda")      # stale: a sequence at position 0 must not read it
    out, at = [], 0
    for n in ((2, 1, 33, 4) if T == 40 else (2, 1, 33, 1, 17, 16)):
        out.append(run_decay(r, slice(at, at + n), dtype, state, i32([(0, n, at, 2)]), qs, silu))
        at += n
    assert at == T
    assert rel(torch.cat(out).view(T, H, dv), want) < 2e-5
    assert rel(state[2], S) < 2e-5 and bool((state[:2] == -9.0).all())


def test_decay_scan_does_not_depend_on_the_batch(cuda):
    """nine sequences of unequal length in one launch against each alone, bit for bit.  The batch is large enough for the
    kernel's wide column groups, a sequence alone is not."""
    H, d, dv = 32, 24, 96
    lens = [1, 17, 2, 16, 33, 5, 1, 20, 9]
    r = decay_inputs(sum(lens), H, d, dv, F32)
    seqs, at = [], 0
    for i, n in enumerate(lens):
        seqs.append((at, n, 0, len(lens) - 1 - i))
        at += n
    state = torch.zeros(len(lens), H, dv, d, device="cuda")
    both = run_decay(r, slice(0, at), F32, state, i32(seqs), 1.0, True)
    for (row0, n, _, slot) in seqs:
        s1 = torch.zeros(1, H, dv, d, device="cuda")
        alone = run_decay(r, slice(row0, row0 + n), F32, s1, i32([(0, n, 0, 0)]), 1.0, True)
        assert torch.equal(both[row0:row0 + n], alone) and torch.equal(state[slot], s1[0])


def test_each_head_decays_by_its_own_number(cuda):
    """one write at token 0, read back for 500 tokens: kept (1), halved, forgotten at once (0), and slowly lost"""
    T, dv, decays = 500, 4, [1.0, 0.5, 0.0, 0.995]
    q, k, v = torch.ones(T, 4, 2), torch.zeros(T, 4, 2), rnd(T, 4, dv, seed=2).float()
    k[0, :, 1] = 1.0
    r = {"q": q, "k": k, "v": v, "decay": torch.tensor(decays)}
    got = run_decay(r, slice(0, T), F32, torch.zeros(1, 4, dv, 2, device="cuda"), i32([(0, T, 0, 0)]), 1.0, False).view(T, 4, dv).cpu().double()
    t = torch.arange(T, dtype=F64)[:, None]
    for h, g in enumerate(decays):
        want = v[0, h].double() * (torch.tensor(g, dtype=F64) ** t)
        assert float((got[:, h] - want).abs().max()) < 2e-5 * float(v[0, h].abs().max()), g


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("H,dv", [(1, 9), (1, 48), (3, 20), (1, 516), (1, 2304), (2, 1001)])
def test_read_out_norm_with_sigmoid_gate(cuda, dtype, H, dv):
    """one norm over all channels (heads=1) or per head; rows a warp takes and rows a whole CTA takes"""
    o, w, gate = rnd(11, H * dv, seed=1), rnd(dv, seed=2), rnd(11, H * dv + 4, seed=3).to(dtype)
    got = _ops().gated_head_norm_rows(dev(o), dev(w), dev(gate, dtype)[:, 4:], heads=H, eps=1e-3, out_dtype=F32,
                                      gate_act=_ops().ACT_SIGMOID)
    want = (O.rms(f32(o).view(11, H, dv), 1e-3) * f32(w)).reshape(11, -1) * torch.sigmoid(gate[:, 4:].double())
    assert rel(got, want) < 1e-5


# ------------------------------------------------------------------------------------------------
# mechanisms alone: residual + Dynamic Tanh norms
# ------------------------------------------------------------------------------------------------
def tanh_norm(cols, seed, alpha):
    w, b = rnd(cols, seed=seed), rnd(cols, seed=seed + 1, scale=0.3)
    return _ops().TanhNorm(alpha, dev(w), dev(b)), lambda x: torch.tanh(float(torch.tensor(alpha)) * x) * f32(w) + f32(b)


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("rows,cols", [(1, 7), (37, 96), (9, 2100), (20, 513), (300, 1032), (3, 4096)])
def test_residual_and_next_norms(cuda, dtype, rows, cols):
    """embedding rows + two norms; two branches, one of them gated per row; routed partials with identity experts; only a
    norm.  The norms' alphas differ, and so do all scales."""
    ops = _ops()
    top, E = 3, 5
    table, ids = rnd(11, cols, seed=1).to(dtype), torch.randint(0, 11, (rows,), generator=torch.Generator().manual_seed(1))
    a, b, h = (rnd(rows, cols + 4, seed=s).to(dtype) for s in (2, 3, 4))
    part = rnd(rows * top, cols, seed=5).float()
    idx = torch.randint(0, E + 3, (rows, top), generator=torch.Generator().manual_seed(2))
    idx[0, 0], idx[-1, -1] = E, E - 1                            # the first identity expert and the last expert
    wt, gate = torch.rand(rows, top, generator=torch.Generator().manual_seed(3)), torch.rand(rows, generator=torch.Generator().manual_seed(4))
    sa, sb = rnd(cols, seed=6), rnd(cols, seed=7)
    (n1, f1), (n2, f2) = tanh_norm(cols, 20, 0.75), tanh_norm(cols, 30, 1.5)
    A, B = a[:, 4:].double(), b[:, :cols].double()
    x = torch.full((rows, cols), float("nan"), device="cuda")
    o1, o2 = ops.tanh_residual_rows(x, [n1, n2], out_dtype=F32, table=dev(table, dtype), ids=ids.int().cuda())
    x0 = table[ids].double()
    assert torch.equal(x.cpu(), table[ids].float()) and rel(o1, f1(x0)) < 1e-5 and rel(o2, f2(x0)) < 1e-5
    kw = dict(a=dev(a, dtype)[:, 4:], a_scale=dev(sa), b_scale=dev(sb), mult=0.3, out_dtype=F32)
    # one branch, no norm
    assert ops.tanh_residual_rows(x, [], a=kw["a"], a_scale=kw["a_scale"], mult=0.3, out_dtype=F32) == []
    x0 = x0 + 0.3 * f32(sa) * A
    assert rel(x, x0) < 1e-6
    # two branches, one norm, in the compute dtype
    o1, = ops.tanh_residual_rows(x, [n2], **dict(kw, out_dtype=BF), b=dev(b, dtype)[:, :cols])
    x0 = x0 + 0.3 * (f32(sa) * A + f32(sb) * B)
    assert o1.dtype == BF and rel(x, x0) < 1e-6 and rel(o1, f2(x0)) < 1e-2
    # gated second branch + routed partials, identity experts read h; rows of identity choices in `part` are never read
    hid = idx >= E
    pn = part.clone()
    pn[hid.reshape(-1)] = float("nan")
    o1, o2 = ops.tanh_residual_rows(x, [n1, n2], **kw, b=dev(b, dtype)[:, :cols], b_gate=dev(gate), part=pn.cuda(), n_partials=top,
                                    idx=idx.int().cuda(), weight=dev(wt), experts=E, h=dev(h, dtype)[:, :cols])
    y = gate.double()[:, None] * B
    for j in range(top):
        y = y + torch.where(hid[:, j:j + 1], wt[:, j:j + 1].double() * h[:, :cols].double(), part.view(rows, top, cols)[:, j].double())
    x0 = x0 + 0.3 * (f32(sa) * A + f32(sb) * y)
    assert rel(x, x0) < 1e-6 and rel(o1, f1(x0)) < 2e-5 and rel(o2, f2(x0)) < 2e-5
    # routed partials alone (no shared expert), every one of them read
    ops.tanh_residual_rows(x, [], **kw, part=part.cuda(), n_partials=top)
    x0 = x0 + 0.3 * (f32(sa) * A + f32(sb) * part.view(rows, top, cols).double().sum(1))
    assert rel(x, x0) < 1e-6
    before = x.clone()
    o1, = ops.tanh_residual_rows(x, [n1], out_dtype=F32)
    assert torch.equal(x, before) and rel(o1, f1(x.cpu().double())) < 1e-5


# ------------------------------------------------------------------------------------------------
# mechanisms alone: router and experts
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("E,top,count,keep", [(14, 3, 2, 1), (12, 4, 4, 2), (9, 1, 9, 1), (16, 5, 8, 4), (6, 6, 1, 1), (40, 8, 5, 3), (1, 1, 1, 1)])
@pytest.mark.parametrize("rows,cols", [(37, 50), (1500, 64)])
def test_softmax_router(cuda, E, top, count, keep, rows, cols):
    """few rows (a CTA each) and many (a warp each); choice values of both signs and all negative; the gate read beside"""
    ops = _ops()
    x, w, gw = rnd(rows, cols, seed=1).to(BF), rnd(E, cols, seed=2, scale=2.0 / cols ** 0.5).float(), rnd(cols, seed=3, scale=0.2).float()
    for shift in (0.0, -3.0):
        corr = (rnd(E, seed=4, scale=0.3) + shift).float()
        r = {"top": top, "scale": 1.7, "groups": {"count": count, "keep": keep}}
        idx, wt = O.route(x.double(), w.double(), corr.double(), r)
        gi, gw_, gate = ops.moe_route_scores(dev(x, BF), dev(w), dev(corr), top, score=ops.SCORE_SOFTMAX, groups=count, keep=keep,
                                             group_top=1, scale=1.7, gate_w=dev(gw))
        assert rel(gate, torch.sigmoid(x.double() @ gw.double())) < 1e-5
        want = torch.zeros(rows, E, dtype=F64).scatter_(1, idx, wt)
        got = torch.zeros(rows, E, dtype=F64).scatter_(1, gi.long().cpu(), gw_.double().cpu())
        same = ((want > 0) == (got > 0)).all(-1)
        assert int((~same).sum()) <= rows // 500                # a tie within fp32 rounding
        assert rel(got[same], want[same]) < 1e-5
        assert all(len(set(row)) == top for row in gi.tolist())
    gi, gw_, gate = ops.moe_route_scores(dev(x, BF), dev(w), None, 1, score=ops.SCORE_SOFTMAX, group_top=1)
    s = torch.softmax(x.double() @ w.double().T, -1)
    assert gate is None and rel(gw_[:, 0], s.amax(-1)) < 1e-5


def test_router_ranks_groups_by_their_largest_choice(cuda):
    """scores made so that the rules differ: group 0 has the largest value, group 1 the two largest together; the correction
    moves the choice but not the weight, also below zero, where a barred expert must not win with 0"""
    ops = _ops()
    x = torch.zeros(2, 8)
    x[:, 0] = 1.0
    w = torch.zeros(6, 8)                          # equal logits: every score is 1 / 6
    for shift in (0.0, -5.0):
        corr = torch.tensor([0.9, 0.1, 0.0, 0.6, 0.5, 0.4]) + shift
        for group_top, first in ((1, 0), (2, 3)):
            idx, wt, _ = ops.moe_route_scores(dev(x), dev(w), dev(corr), 2, score=ops.SCORE_SOFTMAX, groups=2, keep=1, group_top=group_top,
                                              scale=3.0)
            assert sorted(idx[0].tolist()) == [first, first + 1] and rel(wt, torch.full((2, 2), 0.5)) < 1e-6
        idx, _, _ = ops.moe_route_scores(dev(x), dev(w), dev(corr), 3, score=ops.SCORE_SOFTMAX, groups=1, keep=1, group_top=1)
        assert idx[0].tolist() == [0, 3, 4]
        idx, wt, _ = ops.moe_route_scores(dev(x), dev(w), dev(corr), 2, score=ops.SCORE_SIGMOID, groups=2, keep=1, group_top=1)
        assert idx[0].tolist() == [0, 1] and rel(wt, torch.full((2, 2), 0.5)) < 1e-6


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("T", [1, 5, 90])
def test_experts_identity_experts_and_shared_expert(cuda, dtype, T):
    """the model's routed feed-forward alone, through the residual update that adds it up; with every choice an identity
    expert as well"""
    cfg, model = build(config(64, 50, [(lightning(8, 8, [0.5]), moe(6, 6, 4, 24, count=3, keep=2, scale=1.3, shared=40))]), dtype, 3)
    spec, p = cfg["layers"][0]["mlp"], "l0.mlp."
    h = rnd(T, 64, seed=5).to(dtype)
    for all_identity in (False, True):
        if all_identity:
            t = model.state_dict()
            t[p + "correction"] = torch.tensor([0.0] * 6 + [4.0, 5.0, 6.0, 7.0, 8.0, 9.0]).to(BF)
            model.load_weights(t)
        W = {k: v.double() for k, v in model.state_dict().items()}
        L = model.layers[0]
        x = torch.zeros(T, 64, device="cuda")
        zero, one = torch.zeros(64, device="cuda"), torch.ones(64, device="cuda")
        _ops().tanh_residual_rows(x, [], out_dtype=dtype, a=x.clone(), a_scale=zero, b_scale=one, **model._experts(L, dev(h, dtype)))
        want = O.moe_ff(h.double(), W, p, spec)
        assert rel(x, want) < (1e-5 if dtype == F32 else 2e-2)
        if all_identity:
            assert int(O.route(h.double(), W[p + "router"], W[p + "correction"], spec["router"])[0].min()) >= 6


@pytest.mark.parametrize("M,N,K", [(1, 64, 64), (5, 96, 40), (200, 64, 128), (700, 608, 256), (300, 1024, 2048), (5, 54, 33)])
@pytest.mark.parametrize("dtype", [F32, BF])
def test_gelu_gated_unit_and_gelu(cuda, dtype, M, N, K):
    """through the tensor-core epilogues (few and many rows) and the CUDA-core kernel (fp32, odd shapes); pre-activations of
    both signs, far from zero included"""
    ops = _ops()
    x, wg, wu = rnd(M, K, seed=1).to(dtype), rnd(N, K, seed=2, scale=2.0 / K ** 0.5).to(dtype), rnd(N, K, seed=3, scale=2.0 / K ** 0.5).to(dtype)
    wg[0] *= 20.0
    inter = torch.stack([wg, wu], 1).reshape(2 * N, K)
    g, u = x.double() @ wg.double().T, x.double() @ wu.double().T
    got = ops.linear_any(dev(x, dtype), dev(inter, dtype), geglu=True)
    assert got.shape == (M, N) and rel(got, O.gelu_tanh(g) * u) < (1e-5 if dtype == F32 else 1e-2)
    got = ops.linear_any(dev(x, dtype), dev(wu, dtype), act=ops.ACT_GELU_ERF)
    assert rel(got, O.gelu_erf(u)) < (1e-5 if dtype == F32 else 1e-2)
    # the two forms of the function are told apart in fp32
    assert dtype == BF or (rel(O.gelu_tanh(u), O.gelu_erf(u)) > 3e-5 or M * N < 500)


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("M", [1, 7, 90])
def test_capped_logits(cuda, dtype, M):
    ops = _ops()
    x, w = rnd(M, 72, seed=1).to(dtype), rnd(99, 72, seed=2).to(dtype)
    got = ops.glinear(dev(x, dtype), dev(w, dtype), out_dtype=F32, act=ops.ACT_SOFTCAP, act_params=(4.0, 0.0))
    z = x.double() @ w.double().T
    assert float(z.abs().max()) > 12 and rel(got, 4.0 * torch.tanh(z / 4.0)) < 1e-5


# ------------------------------------------------------------------------------------------------
# mechanisms alone: attention
# ------------------------------------------------------------------------------------------------
def rotate_one(u, dims, base, pos):
    out, half = u.clone(), dims // 2
    for i in range(half):
        a = torch.tensor(pos * base ** (-2.0 * i / dims), dtype=F64)
        out[:, i] = u[:, i] * torch.cos(a) - u[:, i + half] * torch.sin(a)
        out[:, i + half] = u[:, i + half] * torch.cos(a) + u[:, i] * torch.sin(a)
    return out


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("rot", [0, 6, 12])
def test_rotation_and_append_of_two_maps(cuda, dtype, rot):
    """each map of each head turns by itself; the pool row is k (two maps per head) | v"""
    ops = _ops()
    H, G, d, dv, T = 4, 2, 12, 20, 9
    row = rnd(T, 2 * (H + G) * d + G * dv + 3, seed=1).to(dtype)
    pos = [0, 1, 2, 63, 64, 65, 1000, 4097, 54321]
    rows = [40, 3, 17, 63, 0, 1, 2, 33, 9]
    inv = torch.tensor([5000.0 ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=F64).cuda() if rot else None
    r = row.double()
    n = 2 * (H + G)
    want = torch.stack([rotate_one(r[t, :n * d].view(n, d), rot, 5000.0, pos[t]) for t in range(T)])
    assert torch.allclose(want[2], O.rotate_halves(r[2, :n * d].view(1, n, d).expand(3, -1, -1), rot, 5000.0)[2])
    pool = torch.zeros(64, G * (2 * d + dv), device="cuda", dtype=dtype)
    q = ops.rope_append(dev(row, dtype), i32(pos), i32(rows), pool, heads=H, kv_heads=G, dim=d, vdim=dv, inv_freq=inv,
                        unit_norm=False, eps=0.0, halves=True, maps=2)
    got = pool[torch.tensor(rows, device="cuda")]
    assert rel(q, want[:, :2 * H].reshape(T, -1)) < 1e-5
    assert rel(got[:, :2 * G * d], want[:, 2 * H:].reshape(T, -1)) < (1e-5 if dtype == F32 else 1e-2)
    assert torch.equal(got[:, 2 * G * d:].cpu(), row[:, n * d:n * d + G * dv])


def attend_direct(q, K, V, pos0, *, scale, window, lam, diff, eps, gate):
    """q [n, H, 2, d] at positions pos0 .., K [ctx, G, 2, d], V [ctx, G, dv] -> [n, H, dv]"""
    n, H = q.shape[:2]
    G = K.shape[1]
    out = torch.zeros(n, H, V.shape[2], dtype=F64)
    for i in range(n):
        lo = max(0, pos0 + i - window + 1) if window else 0
        for h in range(H):
            g = h // (H // G)
            a = [torch.softmax(K[lo:pos0 + i + 1, g, m] @ q[i, h, m] * scale, 0) @ V[lo:pos0 + i + 1, g] for m in (0, 1)]
            out[i, h] = O.combine_maps(a[0], a[1], lam, diff, eps)
            if gate is not None:
                out[i, h] *= torch.sigmoid(gate[i, h])
    return out


def paged(K, V, dtype, pages, page=64):
    """pool whose page pages[k] holds positions 64 k ..; -> (pool, page tables with the sequence in slot 1)"""
    ctx = K.shape[0]
    pool = torch.zeros((max(pages) + 1) * page, K[0].numel() + V[0].numel(), dtype=dtype)
    for j in range(ctx):
        pool[pages[j // page] * page + j % page] = torch.cat([K[j].reshape(-1), V[j].reshape(-1)])
    pt = torch.zeros(2, len(pages) + 3, dtype=torch.int32)
    pt[1, :len(pages)] = torch.tensor(pages)
    return dev(pool, dtype), pt.cuda()


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("H,G,d,dv", [(4, 2, 12, 20), (3, 3, 9, 5), (8, 1, 32, 40), (1, 1, 8, 16), (40, 1, 16, 16), (16, 4, 64, 32), (6, 6, 130, 7),
                                      (4, 4, 8, 260)])
@pytest.mark.parametrize("window", [0, 40])
def test_differential_attention(cuda, dtype, H, G, d, dv, window):
    """portions that start and end inside pages, at page borders and at position 0, shuffled physical pages, prompt tiles
    and decoded rows (1 / 3 key splits) in the same pool"""
    ops = _ops()
    ctx, page = 150, 64
    K, V = rnd(ctx, G, 2, d, seed=1).to(dtype), rnd(ctx, G, dv, seed=2).to(dtype)
    pool, pt = paged(K, V, dtype, [5, 1, 3])
    for pos0, n in ((0, 16), (0, 2), (17, 16), (60, 9), (64, 16), (134, 16), (149, 1), (0, 1), (63, 1), (64, 1)):
        q, gate = rnd(n, H, 2, d, seed=10 + pos0), rnd(n, H + 2, seed=20 + pos0).to(dtype)
        want = attend_direct(f32(q), K.double(), V.double(), pos0, scale=0.4, window=window, lam=0.45, diff=0.2, eps=1e-4, gate=gate.double())
        for ns in ((1, 3) if n == 1 else (1,)):
            got = ops.paged_attention(dev(q.reshape(n, -1)), pool, pt, i32([(0, n, pos0, 1)]), heads=H, kv_heads=G, dim=d, vdim=dv,
                                      page=page, scale=0.4, window=window, diff=(0.45, 0.8, 1e-4), gate=dev(gate, dtype)[:, :H],
                                      max_rows=16 if n > 1 else 1, nsplit=ns, out_dtype=F32)
            assert rel(got.view(n, H, dv), want) < 3e-5, (pos0, n, ns)


def test_two_maps_refuse_what_they_cannot_be_combined_with(cuda):
    ops = _ops()
    pool, pt = paged(rnd(64, 1, 2, 8), rnd(64, 1, 8), F32, [0])
    kw = dict(heads=2, kv_heads=1, dim=8, vdim=8, page=64, scale=1.0, diff=(0.5, 0.5, 1e-5))
    for extra in (dict(sink=torch.zeros(2, device="cuda")), dict(talk=torch.eye(2, device="cuda")), dict(head_scale=torch.ones(2, device="cuda"))):
        with pytest.raises(RuntimeError):
            ops.paged_attention(torch.zeros(1, 32, device="cuda"), pool, pt, i32([(0, 1, 0, 1)]), max_rows=1, **kw, **extra)


@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("window", [0, 2, 63, 64, 65, 72, 300])
def test_window_edges_show(cuda, decode, window):
    """one key of ONE map gets a score far above all others, just inside and just outside the window, at page borders, at the
    first position and ahead of the row: its value must come out exactly when it is seen, with the map's own sign"""
    ops = _ops()
    H, G, d, dv, page, ctx = 2, 1, 16, 8, 64, 450
    K, V = rnd(ctx, G, 2, d, seed=1, scale=0.05), rnd(ctx, G, dv, seed=2)
    big = rnd(d, seed=3)
    big = big / big.norm()
    n, kw = (1 if decode else 5), dict(scale=1.0, window=window, lam=0.7, diff=0.1, eps=1e-6, gate=None)
    for last in (ctx - 1, 383, 384):                      # position of the last row: inside a page, at a page's end and start
        p0 = last - n + 1
        seen_from = max(0, last - window + 1) if window else 0
        places = sorted({seen_from, seen_from - 1, seen_from + 1, 0, 63, 64, 128, 320, last, last - 1, min(last + 1, ctx - 1)} - {-1})
        for m in (0, 1):
            q = torch.zeros(n, H, 2, d, dtype=F64)
            q[:, :, m] = big * 10.0
            for j in places:
                keys = K.clone()
                keys[j, 0, m] = big * 6.0                  # score 60 against 1 at most
                pool, pt = paged(keys, V, F32, list(range(8)))
                want = attend_direct(q, keys, V, p0, **kw)
                got = ops.paged_attention(dev(q.reshape(n, -1)), pool, pt, i32([(0, n, p0, 1)]), heads=H, kv_heads=G, dim=d, vdim=dv, page=page,
                                          scale=1.0, window=window, diff=(0.7, 0.9, 1e-6), max_rows=1 if decode else 16,
                                          nsplit=3 if decode else 1, out_dtype=F32).view(n, H, dv).cpu().double()
                assert rel(got, want) < 1e-4, (last, m, j)
                # a window that is one token off would show
                for edge, off in ((seen_from - 1, 1), (seen_from, -1)):
                    if window > 1 and seen_from > 0 and j == edge:
                        assert rel(attend_direct(q, keys, V, p0, **dict(kw, window=window + off)), want) > 1e-2, (last, m, j)


# ------------------------------------------------------------------------------------------------
# whole models
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_and_layers(cuda, name, dtype):
    from vila_b200.serving import TokenEngine
    cfg, model = build(name, dtype)
    toks = tokens_for(cfg, 150, 1)
    eng = TokenEngine(model, max_tokens=192, slots=1)
    layers, after = [], []
    lg = eng.step([("a", toks, list(range(len(toks))))], layer_outputs=layers)
    want = O.forward(cfg, model.state_dict(), toks, after)
    assert len(layers) == len(after) == len(cfg["layers"])
    for i, (a, b) in enumerate(zip(layers, after)):
        rows_close(a, b, dtype, f"after layer {i}", rare(cfg))
    rows_close(lg, want, dtype, "logits", rare(cfg))
    # a one-token sequence in the slot and pages the long one gave back
    eng.release("a")
    assert rel(eng.step([("b", toks[:1], [0])]), want[:1]) < 2 * tol(dtype)


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_decode_and_portions_match_whole(cuda, name, dtype):
    cfg, model = build(name, dtype, seed=3)
    prompts = {"p": tokens_for(cfg, 140, 2)}
    token_by_token = [[("p", 1)] for _ in range(140)]
    head_then_decode = [[("p", 70)]] + [[("p", 1)] for _ in range(70)]
    portions = [[("p", n)] for n in (2, 3, 2, 57, 1, 16, 17, 2, 33, 5, 2)]
    assert sum(s[0][1] for s in portions) == 140
    for schedule in (token_by_token, head_then_decode, portions):
        got = run_schedule(model, prompts, schedule, max_tokens=192, slots=1)
        check_logits(cfg, model, prompts, got, dtype)


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_mixed_batches_reuse_pages_and_slots(cuda, name, dtype):
    """Four unequal requests share 2 slots and a pool that holds two of them: c and d run in the pages
    and slots a and b gave back; portions sit next to single tokens of the other request."""
    cfg, model = build(name, dtype, seed=4)
    prompts = {"a": tokens_for(cfg, 100, 5), "b": tokens_for(cfg, 37, 6), "c": tokens_for(cfg, 128, 7),
               "d": tokens_for(cfg, 3, 8)}
    schedule = [[("a", 30), ("b", 2)], [("a", 1), ("b", 1)], [("a", 1), ("b", 1)], [("a", 1), ("b", 1)],   # two-row
                [("a", 1), ("b", 30)], [("b", 1), ("a", 47)], [("a", 19), ("b", 1)],   # decode steps: eager, captured, replayed
                [("c", 63)], [("d", 1), ("c", 2)], [("c", 1), ("d", 2)], [("c", 62)]]
    got = run_schedule(model, prompts, schedule, max_tokens=192, slots=2)
    check_logits(cfg, model, prompts, got, dtype)
    if dtype == F32:   # batching must not change a sequence beyond rounding
        alone = run_schedule(model, {"c": prompts["c"]}, [[("c", 128)]], max_tokens=128, slots=1)
        assert rel(got["c"], alone["c"]) < 1e-5


def test_engine_refuses_what_does_not_fit(cuda):
    from vila_b200.serving import TokenEngine
    cfg, model = build("aligned", BF)
    eng = TokenEngine(model, max_tokens=128, slots=1)
    eng.step([("a", tokens_for(cfg, 100, 1), [])])
    with pytest.raises(MemoryError):
        eng.step([("b", [1, 2], [])])           # no slot
    with pytest.raises(MemoryError):
        eng.step([("a", tokens_for(cfg, 40, 2), [])])   # no page
    eng.release("a")
    assert eng.step([("b", [1, 2], [1])]).shape == (1, cfg["vocab"])


def test_a_paused_request_goes_on_where_it_stopped(cuda):
    """a request that is left out of many steps while another is decoded, admitted and released around it"""
    cfg, model = build("odd", F32, seed=10)
    prompts = {"a": tokens_for(cfg, 60, 1), "b": tokens_for(cfg, 45, 2), "c": tokens_for(cfg, 20, 3)}
    schedule = [[("a", 25)], [("b", 40)]] + [[("b", 1)]] * 5 + [[("c", 20)], [("a", 1)], [("a", 34)]]
    check_logits(cfg, model, prompts, run_schedule(model, prompts, schedule, max_tokens=128, slots=2), F32)


def test_long_decode_across_windows_and_page_borders(cuda):
    """300 decoded tokens after a short prompt in fp32: the windows pass over decoded tokens, k | v pages and recurrent
    states are carried across 300 steps (graph replays) and five page borders."""
    cfg, model = build("aligned", F32, seed=5)
    prompts = {"p": tokens_for(cfg, 330, 9)}
    got = run_schedule(model, prompts, [[("p", 30)]] + [[("p", 1)] for _ in range(300)], max_tokens=384, slots=1)
    check_logits(cfg, model, prompts, got, F32)


def test_sharp_attention_in_a_long_window(cuda):
    """With a large score scale the softmax is sharp: every row attends to the best-matching token among up to 600 earlier
    ones, and a window that is one token off would miss some.  Whole prompt, decoded tail, 64-token portions."""
    cfg = json.loads(json.dumps(CONFIGS["ones"]))
    cfg["layers"][4]["mixer"].update(scale=3.0, mask={"size": 600})
    cfg["layers"][1]["mixer"].update(scale=4.0, mask={"size": 129})
    cfg, model = build(cfg, F32, seed=6)
    toks = tokens_for(cfg, 700, 11)
    off = json.loads(json.dumps(cfg))
    off["layers"][4]["mixer"]["mask"]["size"] = 599
    want = O.forward(cfg, model.state_dict(), toks)
    assert rel(O.forward(off, model.state_dict(), toks), want) > 10 * tol(F32)
    for schedule in ([[("p", 700)]], [[("p", 690)]] + [[("p", 1)]] * 10, [[("p", 64)]] * 10 + [[("p", 58)], [("p", 2)]]):
        got = run_schedule(model, {"p": toks}, schedule, max_tokens=704, slots=1)
        rows_close(got["p"], want, F32)


def test_each_part_of_the_weights_reaches_the_logits(cuda):
    """changing one tensor at a time moves the engine's logits as it moves the oracle's (and by more than rounding)"""
    from vila_b200.model import NibelixConfig, NibelixForCausalLM
    cfg, model = build("odd", F32, seed=12)
    base = {k: v.clone() for k, v in model.state_dict().items()}
    toks = tokens_for(cfg, 12, 4)
    whole = [[("p", 10)], [("p", 1)], [("p", 1)]]
    ref = O.forward(cfg, base, toks)
    for n in ["l0.norm1", "l0.norm1.b", "l0.norm1.alpha", "l0.norm2.alpha", "l1.norm2.b", "l0.ls1", "l0.ls2", "l0.mix.lq1", "l0.mix.lk2", "l0.mix.g",
              "l1.mix.norm", "l1.mix.g", "l1.mix.k", "l1.mix.v", "l0.mlp.router", "l0.mlp.correction", "l0.mlp.shared.sg",
              "l0.mlp.shared.up", "l1.mlp.gate", "l1.mlp.up", "l4.mix.v", "final.norm", "final.norm.b", "final.norm.alpha", "head"]:
        w = dict(base)
        w[n] = (base[n].float() * 1.5 + 0.25).to(torch.bfloat16)
        if n.endswith("correction"):                      # another choice, and the weights stay what they were
            w[n] = base[n].flip(0)
        want = O.forward(cfg, w, toks)
        assert rel(want, ref) > 1e-3, n
        m = NibelixForCausalLM(NibelixConfig.from_dict(cfg), "cuda", F32).load_weights(w)
        assert rel(run_schedule(m, {"p": toks}, whole, max_tokens=64, slots=1)["p"], want) < tol(F32), n


def test_each_constant_of_the_configuration_reaches_the_logits(cuda):
    from vila_b200.model import NibelixConfig, NibelixForCausalLM
    cfg, model = build("odd", F32, seed=13)
    W, toks = model.state_dict(), tokens_for(cfg, 60, 4)
    ref = O.forward(cfg, W, toks)

    def at(path, value):
        d = json.loads(json.dumps(cfg))
        o = d
        for k in path[:-1]:
            o = o[k]
        o[path[-1]] = value
        return d
    for path, value in ((("residual_mult",), 0.9), (("logit_softcap",), 3.0), (("logit_softcap",), 0.0), (("norm", "eps"), 0.3),
                        (("layers", 0, "mixer", "diff"), 0.1), (("layers", 0, "mixer", "scale"), 1.5), (("layers", 0, "mixer", "mask", "size"), 36),
                        (("layers", 0, "mixer", "rot", "base"), 50.0), (("layers", 0, "mixer", "rot", "dims"), 4),
                        (("layers", 1, "mixer", "decay"), [0.3, 0.9, 0.99]), (("layers", 0, "mlp", "router", "scale"), 1.0),
                        (("layers", 0, "mlp", "router", "top"), 3), (("layers", 0, "mlp", "router", "groups"), {"count": 3, "keep": 1})):
        d = at(path, value)
        want = O.forward(d, W, toks)
        assert rel(want, ref) > 1e-4, path
        m = NibelixForCausalLM(NibelixConfig.from_dict(d), "cuda", F32).load_weights(W)
        got = run_schedule(m, {"p": toks}, [[("p", 50)]] + [[("p", 1)]] * 10, max_tokens=64, slots=1)["p"]
        assert rel(got, want) < tol(F32), path


def test_generate_through_scheduler_matches_oracle_greedy(cuda):
    """Greedy generation through generate_tokens (continuous batching, chunked prefill, 2 slots for 3
    prompts, small step budget) against greedy decoding with the oracle."""
    from vila_b200.serving import generate_tokens
    cfg, model = build("odd", F32, seed=6)
    prompts = [tokens_for(cfg, n, 10 + n) for n in (41, 5, 70)]
    out = generate_tokens(model, prompts, max_new_tokens=12, slots=2, max_step_tokens=24)
    for p, ids in zip(prompts, out):
        want, margins = O.greedy(cfg, model.state_dict(), p, 12)
        for k, (a, b) in enumerate(zip(ids, want)):
            if margins[k] < 1e-3:
                break       # a tie in the oracle itself
            assert a == b, (k, ids, want)
    # EOS stops a request and frees its slot; sampling with a seed is reproducible
    eos = out[1][3]
    short = generate_tokens(model, prompts[1:2], max_new_tokens=12, eos_token_ids=[eos])
    assert short[0] == out[1][:out[1].index(eos) + 1]
    s1 = generate_tokens(model, prompts[:2], max_new_tokens=6, sample=True, temperature=0.9, top_k=20, top_p=0.9, seed=1)
    s2 = generate_tokens(model, prompts[:2], max_new_tokens=6, sample=True, temperature=0.9, top_k=20, top_p=0.9, seed=1)
    assert s1 == s2 and all(len(s) == 6 for s in s1)
    assert model.generate(prompts[1], max_new_tokens=12)[0] == out[1]


def test_checkpoint_round_trip_and_registry(cuda, tmp_path):
    from vila_b200.model import load_language_model
    from vila_b200.serving import TokenEngine
    cfg, model = build("aligned", BF, seed=7)
    model.save_pretrained(tmp_path / "m")
    again = load_language_model(tmp_path / "m", dtype="bfloat16")
    assert type(again) is type(model) and again.config.to_dict() == model.config.to_dict() == cfg
    toks = tokens_for(cfg, 20, 3)
    a = TokenEngine(model, 64, 1).step([("x", toks, [19])])
    b = TokenEngine(again, 64, 1).step([("x", toks, [19])])
    assert torch.equal(a, b)


def test_command_line_generates_ids(cuda, tmp_path, capsys):
    from llava.cli import infer
    cfg, model = build("ones", F32, seed=8)
    model.save_pretrained(tmp_path / "m")
    prompt = tokens_for(cfg, 9, 4)
    text = infer.main(["--model-path", str(tmp_path / "m"), "--token-ids", ",".join(map(str, prompt)),
                       "--max-new-tokens", "5", "--dtype", "float32"])
    assert [int(t) for t in text.split(",")] == model.generate(prompt, max_new_tokens=5)[0]
    assert text in capsys.readouterr().out


def test_trace_runner_replays_steps(cuda, tmp_path):
    """bin/trace_run on a saved model: three requests over two slots' worth of pages, portions beside
    single tokens, a step that wants nothing, ids released and their pages used again."""
    cfg, model = build("odd", F32, seed=9)
    model.save_pretrained(tmp_path / "m")
    p = {"a": tokens_for(cfg, 70, 1), "b": tokens_for(cfg, 9, 2), "c": tokens_for(cfg, 66, 3)}
    steps = [
        {"step": 0, "entries": [{"id": "a", "tokens": p["a"][:50], "want": [0, 49]}, {"id": "b", "tokens": p["b"][:2], "want": [1]}], "end": []},
        {"step": 1, "entries": [{"id": "b", "tokens": p["b"][2:8], "want": []}], "end": []},
        {"step": 2, "entries": [{"id": "a", "tokens": p["a"][50:51], "want": [0]}, {"id": "b", "tokens": p["b"][8:], "want": [0]}], "end": ["b"]},
        {"step": 3, "entries": [{"id": "a", "tokens": p["a"][51:], "want": [18]}], "end": ["a"]},
        {"step": 4, "entries": [{"id": "c", "tokens": p["c"], "want": [64, 65]}], "end": ["c"]},
    ]
    out = tmp_path / "out"
    r = subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(tmp_path / "m"), "--dtype", "float32",
                        "--out", str(out), "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                       capture_output=True, text=True, timeout=600, cwd=str(ROOT))
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done %d" % k for k in range(5)]
    assert not (out / "1.f32").exists()
    want = {k: O.forward(cfg, model.state_dict(), v) for k, v in p.items()}
    import numpy as np
    rows = {0: [want["a"][0], want["a"][49], want["b"][1]], 2: [want["a"][50], want["b"][8]], 3: [want["a"][69]],
            4: [want["c"][64], want["c"][65]]}
    for k, exp in rows.items():
        got = torch.from_numpy(np.fromfile(out / f"{k}.f32", dtype="<f4").reshape(len(exp), cfg["vocab"]))
        assert rel(got, torch.stack(exp)) < tol(F32), k
