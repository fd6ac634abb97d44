"""Lapilorn on the step engine against the plain float64 oracle (tests/lapilorn_oracle.py): small random models of several
shapes, written to disk as a checkpoint, loaded through the model registry and run through ``HybridSampler.step`` /
``generate`` under different schedules (whole prompts, token by token, portions, mixed batches, reused pages and slots),
and every new mechanism alone against the oracle's function for it."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import lapilorn_oracle as O

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32_TOL = 2e-4
BF16_TOL = 8e-2


# ---- helpers -----------------------------------------------------------------------------------------------------
def _save(tmp_path, cfg, W, name="m"):
    from safetensors.torch import save_file
    d = os.path.join(str(tmp_path), name)
    os.makedirs(d, exist_ok=True)
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in W.items()}, os.path.join(d, "model.safetensors"))
    return d


def _engine(tmp_path, cfg, W, dtype="fp32", pool_tokens=1024, slots=4, name="m", **kw):
    from nanorlhf_b200.models.registry import load_model
    from nanorlhf_b200.sampler.hybrid_sampler import HybridSampler
    path = _save(tmp_path, cfg, W, name)
    model = load_model(path, torch_dtype=torch.float32 if dtype == "fp32" else torch.bfloat16, device="cuda")
    eng = HybridSampler(model, dtype=dtype, max_num_seqs=slots, **kw)
    eng.reset_pool(pool_tokens, slots)
    return eng


def _tokens(cfg, n, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()


def _run_alone(eng, toks, cuts):
    """Feed one sequence in portions ``cuts``; logits of every position."""
    sid = eng.open()
    out, lo = [], 0
    for n in cuts:
        out.append(eng.step([(sid, toks[lo:lo + n], list(range(n)))]).double().cpu())
        lo += n
    eng.close(sid)
    assert lo == len(toks)
    return torch.cat(out)


def _rel(got, want):
    """Worst row error relative to the RMS of the oracle's logits."""
    return ((got - want).pow(2).mean(-1).sqrt().max() / want.pow(2).mean().sqrt()).item()


def _close(got, want, dtype):
    rows = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    if dtype == "fp32":
        return bool(rows.max() < F32_TOL)
    return bool((rows > BF16_TOL).double().mean() <= 0.12 and rows.max() < 3 * BF16_TOL and rows.mean() < 0.5 * BF16_TOL)


def _cuts(total, sizes):
    out, i, k = [], 0, 0
    while i < total:
        n = min(sizes[k % len(sizes)], total - i)
        out.append(n)
        i += n
        k += 1
    return out


def _plan(eng, sids, counts, tokens=None):
    from nanorlhf_b200.sampler.hybrid_sampler import StepPlan
    data, E, T, MB = eng.sched.plan(sids, counts, 0)
    data[:T] = np.zeros(T, dtype=np.int32) if tokens is None else np.asarray(tokens, dtype=np.int32)
    return StepPlan(torch.from_numpy(data).cuda(), E, T, MB)


SHAPES = {
    # both mixers with every feed-forward kind, a borrowing layer, layers of different sizes
    "mixed": dict(layers=("attention/dense", "lightning/moe", "attention/moe", "lightning/dense", "attention/none", "lightning/none", "attention/dense"),
                  kv_from={4: 2, 6: 2}, per_layer={0: dict(heads=6, kv_heads=2, dim=10, vdim=14, scale=0.4, softcap=2.0, rot=dict(base=50.0, dims=10)),
                                                   3: dict(heads=5, dim=6, vdim=4, decay=[0.0, 1.0, 0.5, 0.99, 0.75])}),
    # values that usual defaults make equal or 1: one head, one column, one expert, one group
    "ones": dict(layers=("lightning/moe", "attention/dense"), ff=1, att=dict(heads=1, kv_heads=1, dim=2, vdim=1, scale=1.0, softcap=1.0, rot=dict(base=3.0, dims=2)),
                 lin=dict(heads=1, dim=1, vdim=1, decay=[1.0]), moe=dict(ff=8, experts=1, top=1, scale=1.0, groups=dict(count=1, keep=1), shared=1)),
    # no scaling, no rotation on one layer, no groups, no shared expert, every expert chosen, a width that is no multiple of 8
    "plain": dict(width=44, layers=("attention/moe", "lightning/dense", "attention/none"), att=dict(heads=2, kv_heads=1, dim=6, vdim=6, rot=dict(base=1e4, dims=4)),
                  per_layer={2: dict(rot=None, softcap=None)}, moe=dict(ff=12, experts=3, top=3, groups=None, shared=None)),
    # sizes of a small real model on the tensor-core tiles
    "medium": dict(vocab=1000, width=256, layers=("attention/dense", "lightning/moe", "attention/moe", "lightning/moe"), kv_from={2: 0}, ff=512, limit=3.0,
                   att=dict(heads=8, kv_heads=2, dim=96, vdim=80, scale=0.1, softcap=20.0), lin=dict(heads=4, dim=48, vdim=72),
                   moe=dict(ff=64, experts=16, top=4, groups=dict(count=8, keep=3), shared=128)),
    # an odd width (no vector path anywhere, every GEMM off the tensor-core tiles), tiny feed-forwards, more than 16 heads per key head
    "narrow": dict(width=51, vocab=101, layers=("lightning/moe", "attention/dense", "attention/moe"), ff=30, kv_from={2: 1},
                   att=dict(heads=20, kv_heads=1, dim=8, vdim=8), lin=dict(heads=3, dim=7, vdim=5), moe=dict(ff=10, experts=6, top=2, shared=7)),
    # odd head counts and sizes, expert widths off every tile, groups of one expert
    "odd": dict(vocab=333, width=72, layers=("attention/moe", "lightning/moe", "attention/dense"), ff=100, kv_from={2: 0},
                att=dict(heads=5, kv_heads=5, dim=10, vdim=14, scale=0.2, rot=dict(base=300.0, dims=6, scaling=dict(factor=2.0, low=1.0, high=2.0, original=40))),
                lin=dict(heads=7, dim=10, vdim=14), moe=dict(ff=24, experts=7, top=3, groups=dict(count=7, keep=4), shared=9)),
    # wide heads: key / value columns past the tensor-core kernels, states that need several column slices
    "wide": dict(width=64, layers=("attention/dense", "lightning/moe"), att=dict(heads=2, kv_heads=2, dim=160, vdim=144, scale=0.05),
                 lin=dict(heads=2, dim=136, vdim=160), moe=dict(ff=32, experts=4, top=1, groups=dict(count=2, keep=1))),
}


def _decisive_routers(W):
    """For bf16 runs: a choice of experts that rounding cannot flip.  With random routers some token always has two choice scores nearly
    tied, bf16 rounding of the router's input picks the other one and that token's logits move by far more than rounding.  Here the
    corrections, spread geometrically, decide; the weights stay token dependent.  Token-dependent choices are checked in float32."""
    out = dict(W)
    g = torch.Generator().manual_seed(11)
    for k in W:
        if k.endswith("mlp.correction"):
            out[k] = (-0.3 * 1.5 ** torch.randperm(W[k].shape[0], generator=g).float()).to(W[k].dtype)
        elif k.endswith("mlp.router"):
            out[k] = W[k] * 0.1
    return out


def _model(name, seed=0, dtype="fp32"):
    cfg = O.make_config(**SHAPES[name])
    W = O.random_weights(cfg, seed=seed)
    return cfg, (_decisive_routers(W) if dtype == "bf16" else W)


# ---- mechanisms alone ------------------------------------------------------------------------------------------------
class _HostPlan:
    """A step plan made by hand: entries of ``counts`` tokens that start at positions ``starts`` in state slots ``slots``."""

    def __init__(self, counts, starts, slots, tokens=None):
        i32 = dict(dtype=torch.int32, device="cuda")
        self.E, self.T = len(counts), sum(counts)
        self.cu = torch.tensor([0] + np.cumsum(counts).tolist(), **i32)
        self.tok_entry = torch.tensor(np.repeat(np.arange(len(counts)), counts).tolist(), **i32)
        self.start, self.state_slot = torch.tensor(starts, **i32), torch.tensor(slots, **i32)
        self.tokens = (torch.zeros(self.T) if tokens is None else tokens).int().cuda()


def _lightning_case(H, D, Dv, T, seed, loud=()):
    """Raw projections [T, q | k | v] in whole 32-byte rows; with ``loud`` positions all other keys are (nearly) silent."""
    g = torch.Generator().manual_seed(seed)
    n, nv = H * D, H * Dv
    U = torch.randn(T, (2 * n + nv + 7) // 8 * 8, generator=g)
    if loud:
        quiet = torch.ones(T, dtype=torch.bool)
        quiet[list(loud)] = False
        U[quiet, n:2 * n] = -80.0                            # silu(-80) is about -1e-33
    return U, n, nv


def _lightning_want(U, n, nv, H, decay, state=None, rounded=False):
    act = O.silu(U.double())
    if rounded:
        act = act.float().bfloat16().double()
    T = U.shape[0]
    o, S = O.lightning_core(act[:, :n].reshape(T, H, -1), act[:, n:2 * n].reshape(T, H, -1), act[:, 2 * n:2 * n + nv].reshape(T, H, -1), decay, state)
    return o.reshape(T, -1), S


def _rms(x):
    return x.pow(2).mean().sqrt()


@pytest.mark.parametrize("H,D,Dv", [(2, 64, 64), (3, 128, 128), (1, 32, 24), (2, 16, 72), (2, 40, 8), (1, 96, 120), (3, 12, 12), (2, 5, 7), (1, 1, 1), (1, 200, 130),
                                    (1, 260, 264), (1, 600, 5)])
def test_lightning_scan_continues_from_its_slots(H, D, Dv):
    """Every kernel form, a batch of unequal entries (fresh, carried, in used slots; lengths around a chunk), continued in a second step."""
    from nanorlhf_b200.ops import hybrid as hy
    decay = [0.999, 0.0, 0.5][:H]
    counts, starts, slots = [1, 130, 64, 15, 16, 65, 2], [5, 0, 9, 0, 0, 3, 0], [6, 5, 4, 3, 2, 1, 0]
    counts2 = [70, 1, 17, 63, 2, 16, 1]
    U, n, nv = _lightning_case(H, D, Dv, sum(counts), 1)
    U2, _, _ = _lightning_case(H, D, Dv, sum(counts2), 2)
    st0 = torch.randn(7, H, D, Dv, generator=torch.Generator().manual_seed(3))
    pows = hy.decay_powers(decay, "cuda")
    forms = ["auto", "global"] + (["registers"] if D < 500 else []) + (["chunk"] if D % 8 == 0 and Dv % 8 == 0 and max(D, Dv) <= 128 else [])
    for form in forms:
        chunked = form == "chunk"
        st = st0.clone().cuda()
        got = []
        for u, c, s in ((U, counts, starts), (U2, counts2, [a + b for a, b in zip(starts, counts)])):
            o = torch.full((u.shape[0], nv), float("nan"), device="cuda")
            hy.lightning_scan(u.cuda(), 0, n, 2 * n, pows, st, o, _HostPlan(c, s, slots), False, impl=form)
            got.append(o.double().cpu())
        a = b = 0
        for i in range(7):
            first, second = U[a:a + counts[i]], U2[b:b + counts2[i]]
            # entries of fewer than 16 tokens run token by token in float also beside chunks
            o1, S = _lightning_want(first, n, nv, H, decay, st0[slots[i]].double() if starts[i] else None, chunked and counts[i] >= 16)
            o2, S = _lightning_want(second, n, nv, H, decay, S, chunked and counts2[i] >= 16)
            for o, w in ((got[0][a:a + counts[i]], o1), (got[1][b:b + counts2[i]], o2)):
                assert _rms(o - w) < (6e-3 if chunked else 2e-5) * _rms(w) + 1e-12, (form, i)
                assert (o - w).abs().max() < (3e-2 if chunked else 1e-4) * w.abs().max() + 1e-12, (form, i)
            # given the rounded operands the state is exact: it is never rounded to 16 bits
            assert _rms(st[slots[i]].double().cpu() - S) < (2e-4 if chunked else 1e-5) * _rms(S) + 1e-12, (form, i)
            a, b = a + counts[i], b + counts2[i]


@pytest.mark.parametrize("loud", [(0,), (63,), (64,), (127, 128), (5, 191)])
def test_lightning_chunk_edges(loud):
    """Only a few keys speak: every later token sees them with the right power of the decay, no earlier one does, across chunk edges and
    the edge of a portion."""
    from nanorlhf_b200.ops import hybrid as hy
    H, D, Dv, T = 2, 24, 40, 200
    decay = [0.97, 1.0]
    U, n, nv = _lightning_case(H, D, Dv, T, 7, loud)
    pows = hy.decay_powers(decay, "cuda")
    want, _ = _lightning_want(U, n, nv, H, decay, rounded=True)
    exact, _ = _lightning_want(U, n, nv, H, decay)
    for form, ref in (("chunk", want), ("registers", exact), ("global", exact)):
        for cuts in ([T], [64, 136], [61, 70, 69]):
            st = torch.randn(1, H, D, Dv, device="cuda")     # a used slot
            out, lo = [], 0
            for c in cuts:
                o = torch.empty(c, nv, device="cuda")
                hy.lightning_scan(U[lo:lo + c].cuda(), 0, n, 2 * n, pows, st, o, _HostPlan([c], [lo], [0]), False, impl=form)
                out.append(o.double().cpu())
                lo += c
            got = torch.cat(out)
            assert got[:min(loud)].abs().max() < 1e-20 if min(loud) else True
            err = (got - ref).abs().max(1).values / ref.abs().max(1).values.clamp_min(1e-3 * ref.abs().max())
            assert err.max() < (2e-2 if form == "chunk" else 1e-4), (form, cuts, int(err.argmax()))


def test_lightning_state_is_kept_in_float_over_many_chunks():
    """A slow decay over 40 chunks: 16-bit rounding of the state at every chunk would add up to far more than this."""
    from nanorlhf_b200.ops import hybrid as hy
    H, D, Dv, T = 1, 64, 64, 2560
    U, n, nv = _lightning_case(H, D, Dv, T, 9)
    st, o = torch.zeros(1, H, D, Dv, device="cuda"), torch.empty(T, nv, device="cuda")
    hy.lightning_scan(U.cuda(), 0, n, 2 * n, hy.decay_powers([0.9999], "cuda"), st, o, _HostPlan([T], [0], [0]), True)
    act = O.silu(U.double()).float().bfloat16().double()
    k, v = act[:, n:2 * n], act[:, 2 * n:2 * n + nv]
    S = (k * 0.9999 ** torch.arange(T - 1, -1, -1, dtype=torch.float64)[:, None]).T @ v
    assert _rms(st[0, 0].double().cpu() - S) < 1e-4 * _rms(S)


def _attention_case(tmp_path, dtype, T, needles, seed=0, name="a", borrow=False, **sizes):
    """One attention mixer driven with hand-made projections.  ``needles``: (query position, key position) pairs; the query of head 0 is turned to
    that key (after both rotations), so that this one score stands far above all others where the key is visible."""
    m0 = dict(sizes)
    cfg = O.make_config(layers=("attention/none",) * (2 if borrow else 1), att=m0, kv_from={1: 0} if borrow else None)
    W = O.random_weights(cfg, seed=seed)
    m = cfg["layers"][-1]["mixer"]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    g = torch.Generator().manual_seed(seed + 1)
    q, k = (torch.randn(T, x, D, generator=g, dtype=torch.float64) * 0.5 for x in (H, G))
    v, gate = torch.randn(T, G, Dv, generator=g, dtype=torch.float64), torch.randn(T, H * Dv, generator=g, dtype=torch.float64)
    pos = torch.arange(T)
    for qi, kj in needles:
        k[kj, 0] = k[kj, 0] / k[kj, 0].norm() * D ** 0.5 * 3
        turned = O.rotate_pairs(k[kj:kj + 1], torch.tensor([kj - qi]), m["rot"])[0, 0]       # relative rotation
        q[qi, 0] = turned / turned.norm() * D ** 0.5 * 3
    want = O.attention_core(O.rotate_pairs(q, pos, m["rot"]), O.rotate_pairs(k, pos, m["rot"]), v, m) * torch.sigmoid(gate)

    def run(cuts, pool=1024, gated=True):
        eng = _engine(tmp_path, cfg, W, dtype=dtype, pool_tokens=pool, name=name)
        src, M = eng.layers[0].mixers[0], eng.layers[-1].mixers[0]
        eng.close(eng.open())
        sid = eng.open()
        outs, lo = [], 0
        for n in cuts:
            plan = _plan(eng, [sid], [n])
            for L, mx in ((eng.layers[0], src),) + (((eng.layers[1], M),) if borrow else ()):
                U = torch.zeros(n, L.n_in, device="cuda")
                for nm, x in (("q", q), ("k", k), ("v", v), ("g", gate)):
                    if nm in mx.cols:
                        c0, w = mx.cols[nm]
                        U[:, c0:c0 + w] = x[lo:lo + n].reshape(n, -1).float().cuda()
                out = torch.empty(n, H * Dv, device="cuda", dtype=eng.wdtype)
                eng._rot_attention(mx, U, plan, 1e-5, out)
            outs.append(out.double().cpu())
            lo += n
        eng.close(sid)
        return torch.cat(outs)
    return run, want


NEEDLES = [(300, 2), (47, 47), (15, 16), (17, 17), (31, 32), (200, 15), (255, 256), (320, 319), (329, 1), (100, 101), (64, 63), (128, 64)]


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("borrow", [False, True])
def test_attention_sees_exactly_the_causal_keys(tmp_path, dtype, borrow):
    """Loud keys planted far away, at page and block borders, at the query's own position (the last key it sees) and one position later
    (the first it does not), in whole prompts, in portions and in single-token steps; with own and with another layer's pages."""
    T = 330
    sizes = dict(heads=4, kv_heads=2, dim=16, vdim=24, scale=1.0, softcap=8.0, rot=dict(base=100.0, dims=8, scaling=dict(factor=4.0, low=1.0, high=4.0, original=64)))
    run, want = _attention_case(tmp_path, dtype, T, NEEDLES, borrow=borrow, **sizes)
    tol, scale = (1e-4 if dtype == "fp32" else 4e-2), want.abs().max()
    for cuts in ([T], _cuts(T, [16, 1, 31, 2, 17]), [290] + [1] * 40):
        assert (run(cuts) - want).abs().max() < tol * scale, cuts[:4]
    # the planted keys matter: another key for the same query gives another result
    _, off = _attention_case(tmp_path, dtype, T, [(q, k - 1) for q, k in NEEDLES if 0 < k <= q], **sizes)
    assert all((want[q, :24] - off[q, :24]).abs().max() > 0.1 * scale for q, k in NEEDLES if 0 < k <= q)


@pytest.mark.parametrize("sizes", [dict(heads=1, kv_heads=1, dim=2, vdim=1), dict(heads=6, kv_heads=2, dim=40, vdim=96), dict(heads=8, kv_heads=1, dim=128, vdim=128),
                                   dict(heads=5, kv_heads=5, dim=10, vdim=14), dict(heads=36, kv_heads=2, dim=16, vdim=8), dict(heads=2, kv_heads=1, dim=200, vdim=264),
                                   dict(heads=3, kv_heads=3, dim=7, vdim=9), dict(heads=70, kv_heads=1, dim=8, vdim=16)])
@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
def test_attention_sizes(tmp_path, sizes, dtype):
    """Head counts and sizes on and off every kernel's tile, with the cap and the gate per column."""
    dims = sizes["dim"] // 4 * 2
    run, want = _attention_case(tmp_path, dtype, 150, [(140, 3), (63, 63), (64, 63), (17, 18), (149, 16)], scale=0.3, softcap=3.0,
                                rot=dict(base=1000.0, dims=dims) if dims else None, **sizes)
    for cuts in ([150], [120] + [1] * 30, _cuts(150, [2, 29, 1])):
        err = (run(cuts) - want).abs().max() / want.abs().max()
        assert err < (1e-4 if dtype == "fp32" else 4e-2), cuts[:3]


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
def test_cap_bounds_loud_scores(tmp_path, dtype):
    """Scores far past the cap: without it one key would take everything, with it the others keep their share."""
    sizes = dict(heads=2, kv_heads=1, dim=16, vdim=16, scale=4.0, rot=dict(base=100.0, dims=4))
    run, want = _attention_case(tmp_path, dtype, 80, [(70, 7), (79, 40)], softcap=1.5, **sizes)
    _, uncapped = _attention_case(tmp_path, dtype, 80, [(70, 7), (79, 40)], softcap=None, **sizes)
    assert (want[70, :16] - uncapped[70, :16]).abs().max() > 0.3 * uncapped.abs().max()
    for cuts in ([80], [50] + [1] * 30, [2] * 40):
        assert (run(cuts) - want).abs().max() < (1e-4 if dtype == "fp32" else 3e-2) * want.abs().max()


@pytest.mark.parametrize("impl", ["tile", "simple", "mma"])
def test_gate_per_column_on_every_kernel(impl):
    from nanorlhf_b200 import _C
    from nanorlhf_b200.ops import hybrid as hy
    from nanorlhf_b200.sampler.hybrid_sampler import StepPlan
    H, G, D, T = 6, 2, 32, 50
    g = torch.Generator().manual_seed(2)
    s = _C.StepScheduler(16, 16, 2)
    sid = s.open()
    for counts in ([T], [1]):
        data, E, n, MB = s.plan([sid], counts)
        plan = StepPlan(torch.from_numpy(data).cuda(), E, n, MB)
        for dt in (torch.float32, torch.bfloat16):
            if impl == "mma" and dt == torch.float32:
                continue
            kc, vc = (torch.randn(16, G, 16, D, generator=g).to(dt).cuda() for _ in range(2))
            q, gate = torch.randn(n, H * D, generator=g).cuda(), (torch.randn(n, H * D, generator=g) * 3).cuda()
            a, b = torch.empty(n, H * D, device="cuda", dtype=dt), torch.empty(n, H * D, device="cuda", dtype=dt)
            hy.window_attention(q, kc, vc, plan, 1 << 30, 0.2, 0.7, a, impl=impl, softcap=4.0)
            hy.window_attention(q, kc, vc, plan, 1 << 30, 0.2, 0.7, b, impl=impl, softcap=4.0, gate=gate)
            want = a.double() * torch.sigmoid(gate.double())
            assert (b.double() - want).abs().max() < (1e-6 if dt == torch.float32 else 1.2e-2) * want.abs().max()
            if dt == torch.bfloat16:                         # the float result is gated too
                f = torch.empty(n, H * D, device="cuda")
                if impl == "mma":
                    hy.window_attention(q, kc, vc, plan, 1 << 30, 0.2, 0.7, f, impl=impl, softcap=4.0, gate=gate)
                    assert (f.double() - want).abs().max() < 8e-3 * want.abs().max()


@pytest.mark.parametrize("C", [1, 6, 37, 64, 300, 1540])
@pytest.mark.parametrize("limit", [0.25, 7.0])
def test_clamped_gated_unit(C, limit):
    from nanorlhf_b200.ops import hybrid as hy
    g = torch.Generator().manual_seed(C)
    x = torch.randn(9, 2 * C + 8, generator=g) * 5
    x[0, :2] = torch.tensor([1e4, -1e4])
    for dt, tol in ((torch.float32, 1e-5), (torch.bfloat16, 5e-3)):
        for off in (0, 1):
            out = torch.full((9, C + 8), 5.0, device="cuda", dtype=dt)
            hy.swiglu_cols(x.cuda()[:, off:off + 2 * C], None, out[:, :C], 1.702, limit, 1.0)
            want = O.clamped_glu(x[:, off:off + C].double(), x[:, off + C:off + 2 * C].double(), limit)
            assert (out[:, :C].double().cpu() - want).abs().max() < tol * want.abs().max() and bool((out[:, C:] == 5.0).all())
            hy.swiglu_cols(x.cuda()[:, off:off + 2 * C], None, out[:, :C])      # the plain unit is untouched by the new terms
            want = O.silu(x[:, off:off + C].double()) * x[:, off + C:off + 2 * C].double()
            assert (out[:, :C].double().cpu() - want).abs().max() < tol * want.abs().max()


@pytest.mark.parametrize("n", [3, 48, 255, 256, 2048, 5000])
def test_read_out_norm_over_all_heads(n):
    from nanorlhf_b200.ops import hybrid as hy
    g = torch.Generator().manual_seed(n)
    y, z, w = torch.randn(7, n, generator=g) * 3, torch.randn(7, n + 8, generator=g), torch.rand(n, generator=g) + 0.5
    for dt, tol in ((torch.float32, 1e-5), (torch.bfloat16, 3e-2)):
        out = torch.empty(7, n, device="cuda", dtype=dt)
        hy.gated_part_rmsnorm(y.cuda(), z.cuda()[:, :n], w.cuda(), n, "sigmoid", False, 0.3, 1.0, out)
        want = O.rms(y.double(), 0.3) * w.double() * torch.sigmoid(z[:, :n].double())
        assert (out.double().cpu() - want).abs().max() < tol


@pytest.mark.parametrize("E,top,count,keep,ff", [(1, 1, 1, 1, 8), (6, 2, 3, 2, 12), (8, 4, 2, 1, 7), (12, 3, 12, 5, 16), (40, 6, 8, 3, 32), (320, 9, 20, 4, 4), (6, 6, 3, 3, 5),
                                                 (96, 8, 48, 48, 4)])
def test_sigmoid_routing_by_group_sums(E, top, count, keep, ff):
    """Choice, weights and the dense form's activations; choice scores of both signs; groups of one expert; nothing closed."""
    from nanorlhf_b200.ops import hybrid as hy
    g = torch.Generator().manual_seed(E * 7 + top)
    T = 60
    z, corr = torch.randn(T, E + 3, generator=g) * 2, torch.randn(E, generator=g) * 0.3 - 0.5
    r = dict(experts=E, top=top, scale=1.3, groups=dict(count=count, keep=keep))
    want = [O.route(z[t, :E].double(), corr.double(), r) for t in range(T)]
    ids, wts = torch.empty(T, top, dtype=torch.int32, device="cuda"), torch.empty(T, top, device="cuda")
    gu = torch.randn(T, E * ff, generator=g)
    act = torch.empty(T, E * ff, device="cuda")
    hy.moe_route_all(z.cuda()[:, :E], corr.cuda(), E, top, 1.3, gu=gu.cuda(), ff=ff, act=act, ids=ids, wts=wts, groups=count, keep=keep, sigmoid=True,
                     group_score="top2", relu2=True)
    assert ids.cpu().tolist() == [[e for e, _ in w] for w in want]
    assert (wts.double().cpu() - torch.tensor([[a for _, a in w] for w in want], dtype=torch.float64)).abs().max() < 1e-5
    full = torch.zeros(T, E, dtype=torch.float64)
    for t, w in enumerate(want):
        for e, a in w:
            full[t, e] = a
    ref = full[:, :, None] * torch.relu(gu.double().reshape(T, E, ff)) ** 2
    assert (act.double().cpu().reshape(T, E, ff) - ref).abs().max() < 1e-4
    # the largest member alone as a group's score is another rule
    if 1 < count and keep < count and E // count > 1:
        ids2 = torch.empty_like(ids)
        hy.moe_route_all(z.cuda()[:, :E], corr.cuda(), E, top, 1.3, ids=ids2, wts=wts, groups=count, keep=keep, sigmoid=True)
        assert not torch.equal(ids2, ids)


@pytest.mark.parametrize("W,F,E,top", [(64, 64, 5, 2), (72, 40, 7, 3), (128, 96, 4, 1), (64, 8, 1, 1), (200, 136, 20, 6), (64, 256, 3, 3)])
def test_squared_relu_experts_and_the_weighted_sum_at_the_boundary(W, F, E, top):
    """Rows sorted by expert through two grouped GEMMs, the activation in the first one's epilogue; the boundary gathers the rows with
    their weights on top of the stream and the mixer's result."""
    from nanorlhf_b200.ops import hybrid as hy
    g = torch.Generator().manual_seed(W + F)
    T = 300
    h = torch.randn(T, W, generator=g).bfloat16()
    w = {}
    for e in range(E):
        w[f"e{e}.up"], w[f"e{e}.down"] = ((torch.randn(*s, generator=g) / s[1] ** 0.5).bfloat16() for s in ((F, W), (W, F)))
    ids = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(T)]).int()
    wts = torch.rand(T, top, generator=g) * 2
    want = torch.zeros(T, W, dtype=torch.float64)
    for e in range(E):
        y = O.expert({k: v.double() for k, v in w.items()}, f"e{e}.", h.double())
        want += (wts.double() * (ids == e)).sum(1, keepdim=True) * y
    wu, wd = torch.cat([w[f"e{e}.up"] for e in range(E)]).cuda(), torch.cat([w[f"e{e}.down"] for e in range(E)]).cuda()
    y, slot_of = hy.moe_grouped_ffn(h.cuda(), ids.cuda(), wts.cuda(), wu, wd, E, F, None, relu2=True)
    x, o, w1 = (torch.randn(*s, generator=g) for s in ((T, W), (T, W), (W,)))
    xo, h1 = torch.empty(T, W, device="cuda"), torch.empty(T, W, device="cuda")
    plan = _HostPlan([T], [0], [0])
    hy.parallel_boundary(plan, h.cuda(), 1e-5, x_in=x.cuda(), o=o.cuda(), y=y, slot_of=slot_of, wts=wts.cuda(), w1=w1.cuda(), x_out=xo, h1=h1)
    got = xo.double().cpu() - x.double() - o.double()
    assert (got - want).pow(2).mean().sqrt() < 1e-2 * want.pow(2).mean().sqrt() and (got - want).abs().max() < 4e-2 * want.abs().max()
    assert (h1.double().cpu() - O.rms(xo.double().cpu(), 1e-5) * w1.double()).abs().max() < 2e-5
    out = torch.empty(T, W, device="cuda")                   # and combined by a launch of its own
    hy.moe_grouped_ffn(h.cuda(), ids.cuda(), wts.cuda(), wu, wd, E, F, out, relu2=True)
    assert (out.double().cpu() - got).abs().max() < 1e-4 * want.abs().max()


@pytest.mark.parametrize("shape", ["mixed", "plain", "odd"])
def test_the_stream_after_every_layer(tmp_path, shape):
    cfg, W = _model(shape, seed=2)
    toks = _tokens(cfg, 33, 2)
    keep_want = []
    O.forward(W, cfg, toks, keep=keep_want)
    eng = _engine(tmp_path, cfg, W)
    sid = eng.open()
    got = []
    for lo, hi in ((0, 19), (19, 20), (20, 33)):
        keep = []
        eng._forward_parallel(_plan(eng, [sid], [hi - lo], toks[lo:hi]), [], keep)
        got.append(keep)
    eng.close(sid)
    for i, ref in enumerate(keep_want):
        x = torch.cat([k[i] for k in got]).double().cpu()
        assert (x - ref).abs().max() < 1e-4 * ref.abs().max(), i


def test_borrowed_pages_are_the_source_layers(tmp_path):
    cfg, W = _model("mixed")
    eng = _engine(tmp_path, cfg, W)
    by = {L.spec.index: L.mixers[0] for L in eng.layers}
    assert by[4].k_cache is by[2].k_cache and by[6].v_cache is by[2].v_cache and by[0].k_cache is not by[2].k_cache
    assert "k" not in by[4].cols and "v" not in by[6].cols
    # every layer has one input matrix and one output matrix, feed-forward included
    assert all(L.ff is None for L in eng.layers)



# ---- schedules -----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("shape", list(SHAPES))
def test_prefill_decode_and_portions_agree_with_oracle(tmp_path, shape, dtype):
    cfg, W = _model(shape, dtype=dtype)
    n = 90
    toks = _tokens(cfg, n, 5)
    want = O.forward(W, cfg, toks)
    eng = _engine(tmp_path, cfg, W, dtype=dtype)
    whole = _run_alone(eng, toks, [n])
    assert _close(whole, want, dtype)
    schedules = {"prefill_then_decode": [n - 40] + [1] * 40, "ragged": _cuts(n, [3, 37, 2, 16, 1, 17, 5]), "pairs": [2] * (n // 2)}
    if dtype == "fp32":
        schedules["by_token"] = [1] * n
    for name, cuts in schedules.items():
        got = _run_alone(eng, toks, cuts)
        assert _close(got, want, dtype), name
        assert _close(got, whole, dtype), name


def test_first_tokens_of_a_sequence(tmp_path):
    """One- and two-token sequences: position 0 (no rotation, a single key, an empty state)."""
    cfg, W = _model("mixed")
    eng = _engine(tmp_path, cfg, W)
    for toks in ([5], [5, 5], [0, 96, 3]):
        want = O.forward(W, cfg, toks)
        assert _rel(_run_alone(eng, toks, [len(toks)]), want) < F32_TOL
        assert _rel(_run_alone(eng, toks, [1] * len(toks)), want) < F32_TOL


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("shape", ["mixed", "medium"])
def test_mixed_batches_match_each_request_alone(tmp_path, shape, dtype):
    """Unequal requests share steps (portions beside single tokens, requests that pause); pages and slots are freed and reused."""
    cfg, W = _model(shape, dtype=dtype)
    eng = _engine(tmp_path, cfg, W, dtype=dtype, pool_tokens=16 * 12, slots=3)
    reqs = {name: _tokens(cfg, n, 10 + i) for i, (name, n) in enumerate([("a", 70), ("b", 23), ("c", 1), ("d", 41), ("e", 64), ("f", 9)])}
    want = {k: O.forward(W, cfg, v) for k, v in reqs.items()}
    got, fed, live, waiting = {k: [] for k in reqs}, {k: 0 for k in reqs}, {}, list(reqs)
    portion = {"a": [16, 3, 1, 1, 30, 2, 1, 16], "b": [2, 1, 20], "c": [1], "d": [40, 1], "e": [5, 1, 1, 57], "f": [3, 3, 3]}
    step = 0
    while waiting or live:
        while waiting and len(live) < 3 and eng.sched.num_free_blocks() * 16 >= len(reqs[waiting[0]]) + 16 * len(live):
            live[waiting.pop(0)] = eng.open()
        entries, names = [], []
        for name in list(live):
            if name == "a" and step % 3 == 2:
                continue                                   # a request may sit out a step
            k = portion[name]
            n = min(k[len(got[name]) % len(k)], len(reqs[name]) - fed[name])
            entries.append((live[name], reqs[name][fed[name]:fed[name] + n], list(range(n))))
            names.append((name, n))
        out = eng.step(entries).double().cpu() if entries else None
        o = 0
        for name, n in names:
            got[name].append(out[o:o + n])
            o += n
            fed[name] += n
            if fed[name] == len(reqs[name]):
                eng.close(live.pop(name))
        step += 1
    assert eng.sched.num_open() == 0
    for k in reqs:
        assert _close(torch.cat(got[k]), want[k], dtype), k


def test_long_decoding(tmp_path):
    """Hundreds of single-token steps: the state is carried and the attention keeps every key."""
    cfg, W = _model("odd")
    toks = _tokens(cfg, 260, 8)
    eng = _engine(tmp_path, cfg, W)
    assert _rel(_run_alone(eng, toks, [4] + [1] * 256), O.forward(W, cfg, toks)) < F32_TOL


def test_distant_tokens_reach_through_the_cache_and_the_state(tmp_path):
    """Changing an early token must change late logits, in the engine as in the oracle, in portions and in decoding: through the pages of
    one kind of layer and through the state of the other."""
    for layers, lin in ((("attention/dense", "attention/none"), None), (("lightning/dense", "lightning/none"), dict(heads=2, dim=8, vdim=8, decay=[0.995, 1.0]))):
        cfg = O.make_config(layers=layers, lin=lin)
        W = O.random_weights(cfg, seed=4)
        a = _tokens(cfg, 150, 3)
        b = list(a)
        b[1] = (b[1] + 1) % cfg["vocab"]
        wa, wb = O.forward(W, cfg, a), O.forward(W, cfg, b)
        assert _rel(wa[-8:], wb[-8:]) > 10 * F32_TOL
        eng = _engine(tmp_path, cfg, W)
        for toks, want in ((a, wa), (b, wb)):
            assert _rel(_run_alone(eng, toks, [130] + [1] * 20)[-8:], want[-8:]) < F32_TOL


def test_used_slots_start_from_zero(tmp_path):
    """One slot and few pages: every sequence follows another one's state."""
    cfg, W = _model("mixed")
    eng = _engine(tmp_path, cfg, W, slots=1, pool_tokens=96)
    for seed in (1, 2, 3):
        toks = _tokens(cfg, 80, seed)
        want = O.forward(W, cfg, toks)
        for cuts in ([80], [1] * 80, [2] * 40, _cuts(80, [17, 1, 16, 3])):
            assert _rel(_run_alone(eng, toks, cuts), want) < F32_TOL, cuts[:3]


def test_grouped_and_dense_expert_forms_agree(tmp_path):
    """bf16 serving runs only the chosen experts (rows sorted by expert, the weighted sums formed in the next boundary); the dense form runs
    every expert.  Both against the oracle."""
    for ff in (32, 24):
        cfg = O.make_config(layers=("attention/moe", "lightning/moe"), width=64, moe=dict(ff=ff, experts=6, top=3))
        W = _decisive_routers(O.random_weights(cfg, seed=9))
        toks = _tokens(cfg, 150, 4)
        want = O.forward(W, cfg, toks)
        for form in ("grouped", "dense"):
            eng = _engine(tmp_path, cfg, W, dtype="bf16", name=form, moe=form)
            assert any(L.w_gate_up is not None for L in eng.layers) == (form == "grouped")
            assert _close(_run_alone(eng, toks, [100, 2, 47, 1]), want, "bf16"), (form, ff)


def test_weights_that_change_are_fused_again_without_losing_the_cache(tmp_path):
    cfg, W = _model("mixed")
    eng = _engine(tmp_path, cfg, W)
    toks = _tokens(cfg, 30, 6)
    sid = eng.open()
    eng.step([(sid, toks[:20], [])])
    eng.sync_weights(force=True)
    got = eng.step([(sid, toks[20:], list(range(10)))]).double().cpu()
    eng.close(sid)
    assert _rel(got, O.forward(W, cfg, toks)[20:]) < F32_TOL


# ---- generation through the framework's entry point ------------------------------------------------------------------
class _Tok:
    pad_token_id = 0
    eos_token_id = None


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
def test_greedy_generation_through_the_engine_entry_point(tmp_path, dtype):
    from nanorlhf_b200.models.registry import load_model
    from nanorlhf_b200.sampler.engine import generate, get_native_engine, release_native_engine
    cfg, W = _model("mixed", dtype=dtype)
    path = _save(tmp_path, cfg, W)
    model = load_model(path, torch_dtype=torch.float32 if dtype == "fp32" else torch.bfloat16, device="cuda")
    prompts = [_tokens(cfg, n, 20 + n) for n in (3, 17, 1, 40, 9)]
    new = 24
    out = generate(1, model, _Tok(), prompts, 0.0, new, top_p=1.0, seed=1, rollout_dtype=dtype, max_num_seqs=3,
                   prefill_token_budget=32).cpu()
    far = 0
    for p, row in zip(prompts, out.tolist()):
        full = O.forward(W, cfg, list(p) + row)             # causal: row len(p) - 1 + i decides token i
        for i, t in enumerate(row):
            logits = full[len(p) - 1 + i]
            best = int(logits.argmax())
            if dtype == "fp32":
                assert t == best
            elif t != best and float(logits[best] - logits[t]) > 0.05 * float(logits.std()):
                far += 1                                   # bf16: a near tie of two logits may go the other way
    assert far <= 0.05 * len(prompts) * new
    assert get_native_engine(model, rollout_dtype=dtype).stats["graph_replays"] > 0      # decode steps replay a CUDA graph
    release_native_engine(model)


def test_trace_runner_replays_a_mixed_trace(tmp_path):
    """bin/trace_run as a subprocess: portions beside single tokens, a pool that forces pages and slots to be reused."""
    cfg, W = _model("mixed")
    path = _save(tmp_path, cfg, W)
    reqs = {k: _tokens(cfg, n, 30 + n) for k, n in (("x", 50), ("y", 33), ("z", 2), ("w", 40))}
    steps = [
        {"step": 0, "entries": [{"id": "x", "tokens": reqs["x"][:30], "want": [0, 29]}, {"id": "z", "tokens": reqs["z"], "want": [1]}], "end": ["z"]},
        {"step": 1, "entries": [{"id": "x", "tokens": reqs["x"][30:31], "want": [0]}, {"id": "y", "tokens": reqs["y"][:31], "want": []}], "end": []},
        {"step": 2, "entries": [{"id": "y", "tokens": reqs["y"][31:], "want": [0, 1]}, {"id": "x", "tokens": reqs["x"][31:], "want": [18]}], "end": ["x", "y"]},
        {"step": 3, "entries": [{"id": "w", "tokens": reqs["w"], "want": [39]}], "end": ["w"]},
    ]
    outdir = os.path.join(str(tmp_path), "out")
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", "float32", "--out", outdir,
                        "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True,
                       timeout=900)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == [f"done {i}" for i in range(4)]
    full = {k: O.forward(W, cfg, v) for k, v in reqs.items()}
    want = {0: [full["x"][0], full["x"][29], full["z"][1]], 1: [full["x"][30]], 2: [full["y"][31], full["y"][32], full["x"][49]], 3: [full["w"][39]]}
    for i, rows in want.items():
        got = torch.from_numpy(np.fromfile(os.path.join(outdir, f"{i}.f32"), dtype="<f4").reshape(len(rows), cfg["vocab"])).double()
        assert _rel(got, torch.stack(rows)) < F32_TOL


def test_sampler_command_line_generates_greedily(tmp_path):
    """``python -m nanorlhf_b200.sampler`` on a Lapilorn checkpoint: the class and the engine come from config.json."""
    cfg, W = _model("plain")
    path = _save(tmp_path, cfg, W)
    prompts = [_tokens(cfg, 7, 1), _tokens(cfg, 19, 2)]
    cmd = [sys.executable, "-m", "nanorlhf_b200.sampler", "--model", path, "--dtype", "float32", "--max-tokens", "6"]
    for p in prompts:
        cmd += ["--prompt-ids", ",".join(map(str, p))]
    r = subprocess.run(cmd, capture_output=True, text=True, timeout=900, cwd=ROOT)
    assert r.returncode == 0, r.stderr[-2000:]
    rows = [json.loads(ln) for ln in r.stdout.splitlines() if ln.startswith("{")]
    assert [(x["prompt"], x["sample"]) for x in rows] == [(0, 0), (1, 0)]
    for p, x in zip(prompts, rows):
        full = O.forward(W, cfg, list(p) + x["tokens"])
        assert x["tokens"] == [int(full[len(p) - 1 + i].argmax()) for i in range(6)]
