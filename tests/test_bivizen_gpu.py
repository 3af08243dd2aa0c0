"""Bivizen on the GPU against the plain float64 oracle (oracle/bivizen_oracle.py): every mechanism's kernel
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

from oracle import bivizen_oracle as O

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


# ------------------------------------------------------------------------------------------------
# configurations (none of them a size combination of a published or given model)
# ------------------------------------------------------------------------------------------------
def attention(heads, kv_heads, dim, vdim, rot, *, base=10000.0, softcap=30.0, v_mix=True, scale=None):
    return "attention", {"dim": dim, "heads": heads, "kv_heads": kv_heads, "rot": {"base": base, "dims": rot},
                         "scale": scale if scale is not None else dim ** -0.5, "softcap": softcap, "v_mix": v_mix,
                         "vdim": vdim}


def delta(heads, kv_heads, dim, vdim, conv):
    return "delta", {"conv": conv, "dim": dim, "heads": heads, "kv_heads": kv_heads, "vdim": vdim}


def gla(heads, dim, vdim, tau):
    return "gla", {"dim": dim, "heads": heads, "tau": tau, "vdim": vdim}


def config(width, vocab, layers, eps=1e-5):
    """layers: (mixer, feed-forward size or 0, limit)"""
    return {"architecture": "Bivizen", "layers": [
        {"mixer": m, "mlp": {"ff": ff, "kind": "dense", "limit": lim} if ff else None, "type": t}
        for (t, m), ff, lim in layers], "norm": {"eps": eps}, "vocab": vocab, "width": width}


# name -> (configuration, rank of the decay projections)
CONFIGS = {
    # nothing is a multiple of 8: every projection runs on the CUDA-core kernel in both dtypes; a mixing layer first,
    # one that does not mix between two that do; a layer without feed-forward; a tight limit
    "odd": (config(92, 113, [
        (delta(6, 3, 10, 14, 3), 36, 0.8),
        (attention(4, 2, 12, 20, 6, base=5000.0, softcap=15.0), 20, 3.0),
        (gla(3, 7, 9, 5.0), 0, 0.0),
        (attention(3, 3, 9, 5, 4, v_mix=False), 44, 1.1),
        (attention(6, 2, 16, 20, 16, base=700.0, softcap=4.0), 28, 0.5)]), 5),
    # tensor-core shapes; a recurrent layer first; one key head for 8 query heads; a head rotated in part
    "aligned": (config(128, 256, [
        (gla(4, 32, 48, 12.0), 64, 2.0),
        (delta(8, 2, 64, 32, 4), 160, 7.0),
        (attention(8, 1, 32, 40, 8, base=1e6), 96, 1.0),
        (attention(16, 1, 24, 40, 24, softcap=8.0), 0, 0.0)], eps=1e-6), 16),
    # values that other models make larger: one head, one tap (no tail), tau 1, a feed-forward of one unit, a decay
    # rank of one; a state of 130 key channels; nothing to mix with.  (One value column or one key channel is tested
    # on the kernels: a norm over one or two numbers is nearly their sign, which makes a whole model discontinuous.)
    "ones": (config(64, 97, [
        (delta(1, 1, 130, 11, 1), 8, 1.0),
        (attention(1, 1, 8, 16, 2), 1, 0.3),
        (gla(1, 40, 17, 1.0), 0, 0.0),
        (delta(4, 1, 9, 14, 5), 16, 2.0),
        (gla(2, 6, 10, 30.0), 24, 4.0)]), 1),
    # heads wider than tall and taller than wide, many heads; only recurrent layers: no paged pool at all
    "recurrent": (config(72, 80, [
        (gla(5, 20, 66, 3.0), 24, 2.0),
        (delta(10, 5, 36, 8, 2), 0, 0.0)]), 9),
}


def build(name, dtype, seed=0):
    """name: a key of CONFIGS or a (configuration, decay rank) pair"""
    from vila_b200.model import BivizenConfig, BivizenForCausalLM
    cfg, rank = CONFIGS[name] if isinstance(name, str) else name
    model = BivizenForCausalLM(BivizenConfig.from_dict(cfg), "cuda", dtype).init_random(seed, scale=1.5, decay_rank=rank)
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
    """every row within tolerance (relative to the largest entry of the expected tensor).  bfloat16: the read-out of a
    recurrent head is divided by its own root mean square, so a row whose read-out nearly cancels has the bf16 noise of
    the projections multiplied; one row in `per` may leave the tolerance, none by more than 8 times (a mixer with ONE head
    has nothing to average such a row with: `per` is smaller there).  float32: no exception."""
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
# mechanisms alone: the recurrences
# ------------------------------------------------------------------------------------------------
def unit(u):
    return u / torch.sqrt(u.pow(2).sum(-1, keepdim=True) + 1e-6)


def delta_inputs(T, H, G, d, dv, dtype, seed=0):
    r = {n: rnd(T, *s, seed=seed + i).to(dtype) for i, (n, s) in enumerate(
        (("q", (G, d)), ("k", (G, d)), ("v", (H, dv)), ("a", (H,)), ("b", (H,))))}
    r["A_log"], r["dt_bias"] = rnd(H, seed=seed + 7, scale=0.5).float(), (rnd(H, seed=seed + 8) - 1.5).float()
    return r


def delta_expected(r, q_scale):
    """-> read-outs [T, H, dv], final states [H, dv, d]"""
    G, H = r["q"].shape[1], r["v"].shape[1]
    q, k, v = unit(r["q"].double()) * q_scale, unit(r["k"].double()), r["v"].double()
    beta = torch.sigmoid(r["b"].double())
    g = torch.exp(-torch.exp(r["A_log"].double()) * O.softplus(r["a"].double() + r["dt_bias"].double()))
    out = [O.delta_rule(q[:, h // (H // G)], k[:, h // (H // G)], v[:, h], beta[:, h], g[:, h]) for h in range(H)]
    return torch.stack([o for o, _ in out], 1), torch.stack([S.T for _, S in out])


def run_delta(r, rows, dtype, state, seqs, q_scale):
    """r's rows laid out as a projection leaves them: q | k | v, and decay | step size in a second, wider tensor"""
    T, G, d = r["q"].shape
    H, dv = r["v"].shape[1:]
    qkv = torch.cat([r["q"].reshape(T, -1), r["k"].reshape(T, -1), r["v"].reshape(T, -1), torch.zeros(T, 3, dtype=dtype)], 1)[rows]
    ab = torch.cat([r["a"], torch.zeros(T, 2, dtype=dtype), r["b"]], 1)[rows]
    qkv, ab = dev(qkv, dtype), dev(ab, dtype)
    return _ops().delta_scan(qkv[:, :2 * G * d + H * dv], ab[:, :H], ab[:, H + 2:], state, seqs, heads=H, kv_heads=G, dim=d,
                             vdim=dv, A_log=dev(r["A_log"]), dt_bias=dev(r["dt_bias"]), q_scale=q_scale)


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("H,G,d,dv", [(6, 3, 10, 14), (4, 4, 64, 33), (8, 2, 128, 40), (1, 1, 130, 3), (2, 1, 300, 5), (3, 3, 1, 1),
                                      (2, 2, 32, 128), (64, 16, 16, 320)])
def test_delta_scan_in_portions_through_stale_slots(cuda, dtype, H, G, d, dv):
    T, qs = (40, d ** -0.5) if H == 64 else (70, d ** -0.5)
    r = delta_inputs(T, H, G, d, dv, dtype)
    want, S = delta_expected(r, qs)
    state = torch.full((2, H, dv, d), 55.0, device="cuda")      # stale: a sequence at position 0 must not read it
    out, at = [], 0
    for n in ((1, 2, 21, 16) if T == 40 else (1, 2, 35, 1, 16, 15)):
        out.append(run_delta(r, slice(at, at + n), dtype, state, i32([(0, n, at, 1)]), qs))
        at += n
    assert at == T
    assert rel(torch.cat(out).view(T, H, dv), want) < 2e-5
    assert rel(state[1], S) < 2e-5 and bool((state[0] == 55.0).all())


def gla_inputs(T, H, d, dv, dtype, seed=0):
    r = {n: rnd(T, H, s, seed=seed + i).to(dtype) for i, (n, s) in enumerate((("q", d), ("k", d), ("v", dv), ("z", d)))}
    r["bias"] = rnd(H * d, seed=seed + 9).float()
    return r


def gla_expected(r, q_scale, tau):
    H = r["q"].shape[1]
    z = r["z"].double() + r["bias"].double().view(H, -1)
    alpha = torch.sigmoid(z) ** (1.0 / tau)
    out = [O.gated_linear_rule(r["q"][:, h].double() * q_scale, r["k"][:, h].double(), r["v"][:, h].double(), alpha[:, h])
           for h in range(H)]
    return torch.stack([o for o, _ in out], 1), torch.stack([S.T for _, S in out])


def run_gla(r, rows, dtype, state, seqs, q_scale, tau):
    """q | v | k side by side with gaps, z in a tensor of its own"""
    T, H, d = r["q"].shape
    dv = r["v"].shape[2]
    wide = torch.cat([r["q"].reshape(T, -1), torch.zeros(T, 1, dtype=dtype), r["v"].reshape(T, -1), r["k"].reshape(T, -1)], 1)
    wide, z = dev(wide[rows], dtype), dev(r["z"].reshape(T, -1)[rows], dtype)
    vo = H * d + 1
    return _ops().gla_scan(wide[:, :H * d], wide[:, vo + H * dv:], wide[:, vo:vo + H * dv], z, state, seqs, heads=H, dim=d, vdim=dv,
                           q_scale=q_scale, tau=tau, z_bias=dev(r["bias"]))


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("H,d,dv,tau", [(3, 7, 9, 5.0), (4, 32, 48, 16.0), (2, 128, 64, 1.0), (1, 130, 1, 0.5), (2, 260, 7, 100.0),
                                        (5, 1, 66, 3.0), (64, 12, 320, 8.0)])
def test_gla_scan_in_portions_through_stale_slots(cuda, dtype, H, d, dv, tau):
    T, qs = (40, 0.3) if H == 64 else (70, 0.3)
    r = gla_inputs(T, H, d, dv, dtype)
    want, S = gla_expected(r, qs, tau)
    state = torch.full((3, H, dv, d), -9.0, device="cuda")
    out, at = [], 0
    for n in ((2, 1, 33, 4) if T == 40 else (2, 1, 33, 1, 17, 16)):
        out.append(run_gla(r, slice(at, at + n), dtype, state, i32([(0, n, at, 2)]), qs, tau))
        at += n
    assert at == T
    assert rel(torch.cat(out).view(T, H, dv), want) < 2e-5
    assert rel(state[2], S) < 2e-5 and bool((state[:2] == -9.0).all())


def test_scans_do_not_depend_on_the_batch(cuda):
    """nine sequences of unequal length in one launch against each alone, bit for bit.  The batch is large enough for the
    kernels' wide column groups, a sequence alone is not."""
    H, d, dv = 32, 24, 96
    lens = [1, 17, 2, 16, 33, 5, 1, 20, 9]
    T = sum(lens)
    rd, rg = delta_inputs(T, H, 8, d, dv, F32), gla_inputs(T, H, d, dv, F32, seed=30)
    seqs, at = [], 0
    for i, n in enumerate(lens):
        seqs.append((at, n, 0, len(lens) - 1 - i))
        at += n
    for r, run in ((rd, lambda *a: run_delta(*a, 0.2)), (rg, lambda *a: run_gla(*a, 0.2, 4.0))):
        state = torch.zeros(len(lens), H, dv, d, device="cuda")
        both = run(r, slice(0, T), F32, state, i32(seqs))
        for (row0, n, _, slot) in seqs:
            s1 = torch.zeros(1, H, dv, d, device="cuda")
            alone = run(r, slice(row0, row0 + n), F32, s1, i32([(0, n, 0, 0)]))
            assert torch.equal(both[row0:row0 + n], alone) and torch.equal(state[slot], s1[0])


def test_delta_rule_writes_forgets_and_overwrites(cuda):
    """inputs made so that a fault shows: a full-strength write is read back exactly and survives 400 tokens of other keys
    without decay; a second write under the same key replaces the first; an open decay empties the state"""
    d, dv, T = 16, 8, 420
    r = {"q": torch.zeros(T, 1, d, dtype=F64), "k": torch.zeros(T, 1, d, dtype=F64), "v": rnd(T, 1, dv, seed=1),
         "a": torch.full((T, 1), -200.0, dtype=F64), "b": torch.full((T, 1), 200.0, dtype=F64),
         "A_log": torch.zeros(1), "dt_bias": torch.zeros(1)}
    # key 0 at token 3; keys 1 .. d - 1 in turn afterwards; key 0 again at 410; a full decay at 415
    r["k"][:, 0] = torch.eye(d, dtype=F64)[[0 if t in (3, 410) else 1 + t % (d - 1) for t in range(T)]]
    r["q"][:, 0, 0] = 1.0
    r["a"][415] = 1e4
    want, _ = delta_expected(r, 1.0)
    r32 = {k: v.float() for k, v in r.items()}
    got = run_delta(r32, slice(0, T), F32, torch.zeros(1, 1, dv, d, device="cuda"), i32([(0, T, 0, 0)]), 1.0)
    got = got.view(T, dv).cpu().double()
    v = r["v"][:, 0]
    assert float(got[:3].abs().max()) < 1e-6                    # nothing under key 0 yet
    assert rel(got[3], v[3]) < 1e-5 and rel(got[409], v[3]) < 1e-4     # its own write is seen, and 406 tokens later
    assert rel(got[410], v[410]) < 1e-4 and rel(got[414], v[410]) < 1e-4
    assert float(got[415:].abs().max()) < 1e-6                  # decayed to nothing before token 415's write
    assert rel(got, want.view(T, dv)) < 1e-4


def test_gla_decays_each_key_channel_by_its_own(cuda):
    """channel 0 keeps (z large), channel 1 loses half per token (tau 1, z 0), channel 2 forgets at once (z very negative)"""
    T, dv = 300, 4
    q, k, v = torch.zeros(T, 1, 3), torch.zeros(T, 1, 3), rnd(T, 1, dv, seed=2).float()
    k[0] = 1.0                                                  # one write at token 0 under all three channels
    z = torch.tensor([60.0, 0.0, -300.0]).expand(T, 1, 3)
    for ch, factor in ((0, lambda t: 1.0), (1, lambda t: 0.5 ** t), (2, lambda t: 1.0 if t == 0 else 0.0)):
        q.zero_()
        q[:, 0, ch] = 1.0
        got = run_gla({"q": q, "k": k, "v": v, "z": z, "bias": torch.zeros(3)}, slice(0, T), F32,
                      torch.zeros(1, 1, dv, 3, device="cuda"), i32([(0, T, 0, 0)]), 1.0, 1.0).cpu().double()
        want = torch.stack([v[0, 0].double() * factor(t) for t in range(T)])
        assert float((got - want).abs().max()) < 1e-5 * float(v[0].abs().max())


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("taps", [1, 2, 4, 7])
def test_convolution_of_decoded_tokens_in_one_launch(cuda, dtype, taps):
    """steps that bring one row per sequence (tail and output in one launch) between portions, through stale slots"""
    ops = _ops()
    Cc, lens = 37, {"a": 29, "b": 12}
    w = rnd(Cc, taps, seed=1, scale=0.5)
    u = {k: rnd(n, Cc, seed=3 + i).to(dtype) for i, (k, n) in enumerate(lens.items())}
    want = {k: O.silu(O.causal_conv(u[k].double(), w)) for k in u}
    state = torch.full((3, taps - 1, Cc), 77.0, device="cuda") if taps > 1 else None
    slot, at, got = {"a": 2, "b": 0}, {"a": 0, "b": 0}, {"a": [], "b": []}
    plan = [[("a", 1), ("b", 1)], [("b", 1)], [("b", 1), ("a", 1)], [("a", 9), ("b", 3)], [("a", 1), ("b", 1)], [("b", 1), ("a", 1)],
            [("a", 2)]] + [[("a", 1)]] * 10 + [[("b", 4), ("a", 4)]]
    for step in plan:
        rows, seqs, row_seq = [], [], []
        for k, n in step:
            seqs.append((len(rows), n, at[k], slot[k]))
            row_seq += [len(seqs) - 1] * n
            rows += list(u[k][at[k]:at[k] + n])
        wide = torch.zeros(len(rows), Cc + 5, dtype=dtype)
        wide[:, 3:3 + Cc] = torch.stack(rows)
        out = ops.causal_conv_rows(dev(wide, dtype)[:, 3:3 + Cc], dev(w), None, state, i32(seqs), i32(row_seq),
                                   act=ops.CONV_SILU, out_dtype=F32)
        o = 0
        for k, n in step:
            got[k].append(out[o:o + n].cpu())
            at[k] += n
            o += n
    for k in u:
        assert at[k] == lens[k] and rel(torch.cat(got[k]), want[k]) < 1e-5, k


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("H,dv", [(3, 9), (4, 48), (1, 1), (2, 300)])
def test_gated_head_norm(cuda, dtype, H, dv):
    o, w, gate = rnd(11, H * dv, seed=1), rnd(dv, seed=2), rnd(11, H * dv + 4, seed=3).to(dtype)
    got = _ops().gated_head_norm_rows(dev(o), dev(w), dev(gate, dtype)[:, 4:], heads=H, eps=1e-3, out_dtype=F32)
    want = (O.rms(o.float().double().view(11, H, dv), 1e-3) * w.float().double()).reshape(11, -1) * O.silu(gate[:, 4:].double())
    assert rel(got, want) < 1e-5


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("rows,cols", [(1, 7), (37, 96), (9, 2100), (20, 513), (300, 1032), (3, 4096), (3, 8192), (2, 9000)])
def test_scaled_residual_and_next_norm(cuda, dtype, rows, cols):
    ops = _ops()
    x0, a, b = rnd(rows, cols, seed=1), rnd(rows, cols, seed=2).to(dtype), rnd(rows, cols, seed=3).to(dtype)
    sa, sb, w = rnd(cols, seed=4), rnd(cols, seed=5), rnd(cols, seed=6)
    f = lambda t: t.float().double()
    x = dev(x0)
    h = ops.scaled_residual_norm_rows(x, dev(a, dtype), dev(sa), dev(b, dtype), dev(sb), dev(w), 1e-3, out_dtype=F32)
    want = f(x0) + f(sa) * a.double() + f(sb) * b.double()
    assert rel(x, want) < 1e-6 and rel(h, O.rms(want, 1e-3) * f(w)) < 1e-5
    x = dev(x0)
    wide = dev(torch.cat([a, b], 1), dtype)     # a branch that is a column slice of a wider tensor; no second branch, no norm
    assert ops.scaled_residual_norm_rows(x, wide[:, :cols], dev(sa)) is None
    assert rel(x, f(x0) + f(sa) * a.double()) < 1e-6
    x = dev(x0)
    hb = ops.scaled_residual_norm_rows(x, dev(a, dtype), dev(sa), w=dev(w), eps=1e-3, out_dtype=BF)
    assert hb.dtype == BF and rel(hb, O.rms(f(x0) + f(sa) * a.double(), 1e-3) * f(w)) < 1e-2


# ------------------------------------------------------------------------------------------------
# mechanisms alone: attention and the feed-forward
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("rot", [0, 6, 12])
def test_rotation_value_mixing_and_append(cuda, dtype, rot):
    ops = _ops()
    H, G, d, dv, T, lam = 4, 2, 12, 20, 9, 0.37
    row, vf = rnd(T, (H + G) * d + G * dv + 3, seed=1).to(dtype), rnd(T, G * dv + 5, seed=2).to(dtype)
    pos = [0, 1, 2, 63, 64, 65, 1000, 4097, 54321]
    rows = [40, 3, 17, 63, 0, 1, 2, 33, 9]
    inv = torch.tensor([5000.0 ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=F64).cuda() if rot else None
    r = row.double()
    want = torch.stack([rotate_one(r[t, :(H + G) * d].view(H + G, d), rot, 5000.0, pos[t]) for t in range(T)])
    assert torch.allclose(want[2], O.rotate_halves(r[2, :(H + G) * d].view(1, H + G, d).expand(3, -1, -1), rot, 5000.0)[2])
    for mix in (True, False):
        pool = torch.zeros(64, G * (d + dv), device="cuda", dtype=dtype)
        kw = dict(v_first=dev(vf, dtype)[:, 5:], v_mix=lam) if mix else {}
        q = ops.rope_append(dev(row, dtype), i32(pos), i32(rows), pool, heads=H, kv_heads=G, dim=d, vdim=dv, inv_freq=inv,
                            unit_norm=False, eps=0.0, halves=True, **kw)
        v = r[:, (H + G) * d:(H + G) * d + G * dv]
        if mix:
            v = (1 - lam) * v + lam * vf[:, 5:].double()
        got = pool[torch.tensor(rows, device="cuda")]
        assert rel(q, want[:, :H].reshape(T, -1)) < 1e-5
        assert rel(got[:, :G * d], want[:, H:].reshape(T, -1)) < (1e-5 if dtype == F32 else 1e-2)
        assert rel(got[:, G * d:], v) < (1e-6 if dtype == F32 else 1e-2)


def rotate_one(u, dims, base, pos):
    out, half = u.clone(), dims // 2
    for i in range(half):
        a = torch.tensor(pos * base ** (-2.0 * i / dims), dtype=F64)
        out[:, i] = u[:, i] * torch.cos(a) - u[:, i + half] * torch.sin(a)
        out[:, i + half] = u[:, i + half] * torch.cos(a) + u[:, i] * torch.sin(a)
    return out


def attend_direct(q, K, V, pos0, *, scale, cap, gate):
    """q [n, H, d] at positions pos0 .., K [ctx, G, d], V [ctx, G, dv] -> [n, H, dv]"""
    n, H, _ = q.shape
    G = K.shape[1]
    out = torch.zeros(n, H, V.shape[2], dtype=F64)
    for i in range(n):
        for h in range(H):
            s = O.softcap(K[:pos0 + i + 1, h // (H // G)] @ q[i, h] * scale, cap)
            out[i, h] = torch.softmax(s, 0) @ V[:pos0 + i + 1, h // (H // G)]
            if gate is not None:
                out[i, h] *= torch.sigmoid(gate[i, h])
    return out


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("H,G,d,dv", [(4, 2, 12, 20), (3, 3, 9, 5), (8, 1, 32, 40), (1, 1, 8, 16), (40, 1, 16, 16), (32, 8, 64, 32), (6, 6, 130, 7)])
def test_attention_with_capped_scores_and_gate(cuda, dtype, H, G, d, dv):
    """portions that start and end inside pages, at page borders and at position 0, shuffled physical pages, prompt tiles
    and decoded rows (1 / 3 key splits) in the same pool; scores well beyond the cap"""
    ops = _ops()
    ctx, page, cap = 150, 64, 2.5
    K, V = rnd(ctx, G, d, seed=1).to(dtype), rnd(ctx, G, dv, seed=2).to(dtype)
    pages = [5, 1, 3]
    pool = torch.zeros(6 * page, G * (d + dv), dtype=dtype)
    for j in range(ctx):
        pool[pages[j // page] * page + j % page] = torch.cat([K[j].reshape(-1), V[j].reshape(-1)])
    pt = torch.zeros(2, 6, dtype=torch.int32)
    pt[1, :3] = torch.tensor(pages)
    for pos0, n in ((0, 16), (0, 2), (17, 16), (60, 9), (64, 16), (134, 16), (149, 1), (0, 1), (63, 1), (64, 1)):
        q, gate = rnd(n, H, d, seed=10 + pos0), rnd(n, H + 2, seed=20 + pos0).to(dtype)
        want = attend_direct(q.float().double(), K.double(), V.double(), pos0, scale=0.9, cap=cap, gate=gate.double())
        for ns in ((1, 3) if n == 1 else (1,)):
            got = ops.paged_attention(dev(q.reshape(n, -1)), dev(pool, dtype), pt.cuda(), i32([(0, n, pos0, 1)]), heads=H, kv_heads=G,
                                      dim=d, vdim=dv, page=page, scale=0.9, softcap=cap, gate=dev(gate, dtype)[:, :H],
                                      max_rows=16 if n > 1 else 1, nsplit=ns, out_dtype=F32)
            assert rel(got.view(n, H, dv), want) < 2e-5, (pos0, n, ns)


@pytest.mark.parametrize("decode", [False, True])
def test_far_keys_page_borders_and_the_cap_show(cuda, decode):
    """one key gets a score far above all others, hundreds of positions back, at the first position and on both sides of a
    page border: its value must come out, in tiles and in decoded rows.  Two keys of very different raw scores, both beyond the cap,
    must share the weight; without the cap the larger one takes it all.  A key after the row must not be seen."""
    ops = _ops()
    H, G, d, dv, page, ctx = 2, 1, 16, 8, 64, 700
    K, V = rnd(ctx, G, d, seed=1, scale=0.1), rnd(ctx, G, dv, seed=2)
    big = rnd(d, seed=3)
    big = big / big.norm()
    pt = torch.arange(11, dtype=torch.int32)[None].cuda()
    n = 1 if decode else 5

    def run(keys, cap, end=ctx):
        pool = torch.cat([keys.reshape(ctx, -1), V.reshape(ctx, -1)], 1)
        pool = torch.cat([pool, torch.zeros(704 - ctx, G * (d + dv), dtype=F64)])
        q = (big * 10.0).expand(n, H, d).reshape(n, -1)
        return ops.paged_attention(dev(q), dev(pool), pt, i32([(0, n, end - n, 0)]), heads=H, kv_heads=G, dim=d, vdim=dv, page=page,
                                   scale=1.0, softcap=cap, max_rows=1 if decode else 16, nsplit=3 if decode else 1,
                                   out_dtype=F32).view(n, H, dv).cpu().double()

    for j in (0, 1, 13, 63, 64, 127, 128, 500, 639, 640, ctx - n):
        keys = K.clone()
        keys[j, 0] = big * 6.0                    # score 60; with the cap of 25: 24.6 against 2 at most
        for cap in (0.0, 25.0):
            assert rel(run(keys, cap), V[j, 0].expand(n, H, dv)) < 1e-4, (j, cap)
    keys = K.clone()
    keys[100, 0], keys[300, 0] = big * 6.0, big * 9.0
    assert rel(run(keys, 0.0), V[300, 0].expand(n, H, dv)) < 1e-4
    e = torch.exp(15.0 * torch.tanh(torch.tensor([60.0, 90.0], dtype=F64) / 15.0))
    assert rel(run(keys, 15.0), ((e[0] * V[100, 0] + e[1] * V[300, 0]) / e.sum()).expand(n, H, dv)) < 1e-2
    keys = K.clone()
    keys[650, 0] = big * 6.0                      # rows end at 640: this one lies ahead of them
    q = (big * 10.0).expand(n, H, d)
    assert rel(run(keys, 25.0, end=640), attend_direct(q, keys, V, 640 - n, scale=1.0, cap=25.0, gate=None)) < 1e-4


@pytest.mark.parametrize("M,N,K", [(1, 64, 64), (5, 96, 40), (200, 64, 128), (700, 608, 256), (300, 1024, 2048), (5, 54, 33)])
@pytest.mark.parametrize("dtype", [F32, BF])
def test_clamped_gated_unit(cuda, dtype, M, N, K):
    """through the tensor-core epilogues (few and many rows), the CUDA-core kernel (fp32, odd shapes); pre-activations on both
    sides of the limit, far below zero included"""
    ops = _ops()
    x, wg, wu = rnd(M, K, seed=1).to(dtype), rnd(N, K, seed=2, scale=2.0 / K ** 0.5).to(dtype), rnd(N, K, seed=3, scale=2.0 / K ** 0.5).to(dtype)
    wg[0] *= 40.0
    inter = torch.stack([wg, wu], 1).reshape(2 * N, K)
    got = ops.linear_any(dev(x, dtype), dev(inter, dtype), glu_clamp=(1.702, 1.3))
    g = torch.clamp_max(x.double() @ wg.double().T, 1.3)
    u = torch.clamp(x.double() @ wu.double().T, -1.3, 1.3)
    assert got.shape == (M, N) and rel(got, g * torch.sigmoid(1.702 * g) * (u + 1.0)) < (1e-5 if dtype == F32 else 1e-2)


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


def test_long_decode_across_page_borders(cuda):
    """300 decoded tokens after a short prompt in fp32: k | v pages, convolution tails and recurrent states are
    carried across 300 steps (graph replays) and five page borders."""
    cfg, model = build("aligned", F32, seed=5)
    prompts = {"p": tokens_for(cfg, 330, 9)}
    got = run_schedule(model, prompts, [[("p", 30)]] + [[("p", 1)] for _ in range(300)], max_tokens=384, slots=1)
    check_logits(cfg, model, prompts, got, F32)


def test_sharp_attention_over_a_long_context(cuda):
    """With a large score scale and cap the softmax is sharp: every row attends to the best-matching token among up to
    700 earlier ones.  Whole prompt, decoded tail, 64-token portions."""
    cfg, rank = json.loads(json.dumps(CONFIGS["ones"]))
    cfg["layers"][1]["mixer"].update(scale=4.0, softcap=60.0)
    cfg, model = build((cfg, rank), F32, seed=6)
    toks = tokens_for(cfg, 700, 11)
    for schedule in ([[("p", 700)]], [[("p", 690)]] + [[("p", 1)]] * 10, [[("p", 64)]] * 10 + [[("p", 58)], [("p", 2)]]):
        got = run_schedule(model, {"p": toks}, schedule, max_tokens=704, slots=1)
        check_logits(cfg, model, {"p": toks}, got, F32)


def test_each_part_of_the_weights_reaches_the_logits(cuda):
    """changing one tensor at a time moves the engine's logits as it moves the oracle's (and by more than rounding), except
    the first mixing layer's unused mixing number"""
    from vila_b200.model import BivizenConfig, BivizenForCausalLM
    cfg, model = build("odd", F32, seed=12)
    base = {k: v.clone() for k, v in model.state_dict().items()}
    toks = tokens_for(cfg, 12, 4)
    whole = [[("p", 10)], [("p", 1)], [("p", 1)]]
    ref = O.forward(cfg, base, toks)
    picks = ["l1.mix.q.b", "l1.mix.v.b", "l1.mix.g", "l4.mix.vmix", "l0.mix.q.conv", "l0.mix.v.conv", "l0.mix.A_log", "l0.mix.dt_bias",
             "l0.mix.norm", "l0.mix.b", "l2.mix.a1", "l2.mix.a2", "l2.mix.a2.b", "l2.mix.norm", "l2.ls1", "l3.ls2", "l0.mlp.up", "final.norm"]
    for n in picks + ["l1.mix.vmix"]:
        w = dict(base)
        w[n] = (base[n].float() * 1.5 + 0.25).to(torch.bfloat16)
        want = O.forward(cfg, w, toks)
        moved = rel(want, ref)
        assert (moved == 0.0) if n == "l1.mix.vmix" else moved > 2e-3, (n, moved)
        m = BivizenForCausalLM(BivizenConfig.from_dict(cfg), "cuda", F32).load_weights(w)
        assert rel(run_schedule(m, {"p": toks}, whole, max_tokens=64, slots=1)["p"], want) < tol(F32), n


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
