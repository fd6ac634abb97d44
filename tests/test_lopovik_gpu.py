"""Lopovik on the step engine against the plain float64 oracle (tests/lopovik_oracle.py): small random models of several
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

import lopovik_oracle as O

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
    # every feed-forward kind, a loop over layers of different sizes in the middle
    "mixed": dict(ffs=("dense", "moe", None, "moe", "dense"), loop=(1, 4, 2),
                  per_layer={2: dict(heads=2, dim=4, rot_dim=8, vdim=6, kv_rank=12, q_rank=8, scale=0.25, base=500.0),
                             4: dict(heads=5, dim=12, rot_dim=2, vdim=8, kv_rank=24, q_rank=40, scale=0.2, base=50.0)}),
    # values that usual defaults make equal or 1: one head, one query latent column, one expert, one pass, a loop at layer 0
    "ones": dict(ffs=("moe", "dense"), loop=(0, 1, 1), dense_ff=1, att=dict(heads=1, dim=1, rot_dim=2, vdim=1, kv_rank=8, q_rank=1, scale=1.0),
                 moe=dict(ff=8, experts=1, top=1)),
    # no loop, every expert chosen, a width that is no multiple of 8
    "plain": dict(width=44, ffs=("moe", "dense", None), loop=None, att=dict(heads=2, dim=6, rot_dim=8, vdim=6, kv_rank=10, q_rank=14),
                  moe=dict(ff=12, experts=3, top=3)),
    # sizes of a small real model: wide latent (key rows past 128 columns), many experts, sizes on the GEMM tiles; all layers loop
    "medium": dict(vocab=1000, width=256, ffs=("dense", "moe", "moe"), loop=(0, 3, 2), dense_ff=512,
                   att=dict(heads=8, dim=32, rot_dim=16, vdim=48, kv_rank=160, q_rank=128, scale=0.12, base=5e5), moe=dict(ff=64, experts=8, top=2)),
    # a width that is odd (no vector path anywhere, every GEMM off the tensor-core tiles), tiny feed-forwards, the loop at the end
    "narrow": dict(width=51, vocab=101, ffs=("moe", "dense", "moe"), loop=(1, 3, 3), dense_ff=30, moe=dict(ff=10, experts=3, top=2)),
    # odd head counts and sizes (key rows of 4 k + 2 columns run on the one-query kernel), expert widths off the fused epilogue
    "odd": dict(vocab=333, width=72, ffs=("moe", "dense", "moe"), loop=(0, 2, 2), dense_ff=100, moe=dict(ff=24, experts=7, top=3),
                att=dict(heads=5, dim=10, rot_dim=6, vdim=14, kv_rank=20, q_rank=13, scale=0.2, base=300.0)),
    # the widest rows the tensor-core kernels take, more than 16 heads
    "wide": dict(width=64, ffs=("dense", "moe"), loop=(1, 2, 2), moe=dict(ff=32, experts=4, top=1),
                 att=dict(heads=18, dim=8, rot_dim=64, vdim=16, kv_rank=512, q_rank=32, scale=0.15)),
}


def _decisive_routers(W):
    """For bf16 runs: a choice of experts that rounding cannot flip.  With random routers some token always has two scores nearly
    tied, bf16 rounding of the router's input picks the other one and that token's logits move by far more than rounding.  Here
    column 0 of the stream is a constant that no layer changes and the router reads mostly that column, with well separated rows;
    the scores stay token dependent through the norm and a small rest.  Token-dependent choices are checked in float32."""
    out = dict(W)
    g = torch.Generator().manual_seed(11)
    n = W["embed"].shape[1]
    out["embed"] = W["embed"].clone()
    out["embed"][:, 0] = 2.0
    for k in W:
        if k.endswith(".o") or k.endswith(".down"):
            out[k] = W[k].clone()
            out[k][0] = 0
        elif k == "loop.in":
            out[k] = W[k].clone()
            out[k][0] = 0
            out[k][0, n] = 1.0
        elif k.endswith("mlp.router"):
            E = W[k].shape[0]
            out[k] = W[k] * 0.05
            out[k][:, 0] = ((torch.randperm(E, generator=g).float() + 1) / E * 3.0 - 1.5).to(W[k].dtype)
        elif k.endswith("norm2"):
            out[k] = W[k].clone()
            out[k][0] = 0.5
    return out


def _model(name, seed=0, dtype="fp32"):
    cfg = O.make_config(**SHAPES[name])
    W = O.random_weights(cfg, seed=seed)
    return cfg, (_decisive_routers(W) if dtype == "bf16" else W)


# ---- mechanisms alone ------------------------------------------------------------------------------------------------
class _HostPlan:
    """A step plan made by hand: entries of ``counts`` tokens that start at positions ``starts`` in state slots ``slots``."""

    def __init__(self, counts, starts, slots, tokens):
        i32 = dict(dtype=torch.int32, device="cuda")
        self.cu = torch.tensor([0] + np.cumsum(counts).tolist(), **i32)
        self.tok_entry = torch.tensor(np.repeat(np.arange(len(counts)), counts).tolist(), **i32)
        self.start, self.state_slot = torch.tensor(starts, **i32), torch.tensor(slots, **i32)
        self.tokens = tokens.int().cuda()


@pytest.mark.parametrize("W,counts", [(44, [5, 1, 9]), (51, [3, 2]), (1028, [1, 1, 4]), (516, [3, 1]), (4104, [2, 3]), (4096, [1, 2]), (12, [700, 1, 1360]), (12, [4096, 3]), (20, [1, 8000, 300])])
def test_boundary_adds_norms_and_shifts(W, counts):
    """Sum of stream, result and gathered expert rows; both norms; the shift inside an entry, at its first token (zeros or the slot's
    row) and across the rows of different blocks (one to six tokens per block); what is carried and what is handed over."""
    from nanorlhf_b200.ops import hybrid as hy
    g = torch.Generator().manual_seed(W)
    E, T, eps, top = len(counts), sum(counts), 1e-5, 2
    starts = [0 if e % 2 == 0 else 7 for e in range(E)]
    slots = list(range(E))[::-1]
    emb, tok = torch.randn(30, W, generator=g), torch.randint(0, 30, (T,), generator=g)
    plan = _HostPlan(counts, starts, slots, tok)
    x, o, y = torch.randn(T, W, generator=g), torch.randn(T, W, generator=g), torch.randn(T * top, W, generator=g)
    perm = torch.randperm(T * top, generator=g)
    w1, w2, mu = torch.rand(W, generator=g) + 0.5, torch.rand(W, generator=g) + 0.5, torch.rand(W, generator=g)
    state, prev_carry = torch.randn(E + 1, W, generator=g), torch.randn(E, W, generator=g)
    total = x.double() + o.double() + y.double()[perm].reshape(T, top, W).sum(1)
    n = O.rms(total, eps)
    want1 = torch.empty(T, W, dtype=torch.float64)
    lo = 0
    for e, c in enumerate(counts):
        h = n[lo:lo + c] * w1.double()
        above = torch.cat([state[slots[e]].double()[None] if starts[e] else torch.zeros(1, W, dtype=torch.float64), h[:-1]])
        want1[lo:lo + c] = h + (above - h) * mu.double()
        lo += c
    last = torch.tensor(np.cumsum(counts) - 1)
    for hd, tol in ((torch.float32, 2e-5), (torch.bfloat16, 4e-2)):
        f32 = dict(dtype=torch.float32, device="cuda")
        xo, raw, h1, h2 = torch.empty(T, W, **f32), *(torch.empty(T, W, dtype=hd, device="cuda") for _ in range(3))
        carry, old = torch.full((E, W), 7.0, **f32), torch.zeros(E + 1, W, **f32)
        hy.parallel_boundary(plan, emb.cuda(), eps, x_in=x.cuda(), o=o.cuda(), y=y.cuda(), slot_of=perm.int().cuda(), w1=w1.cuda(), w2=w2.cuda(),
                             mu=mu.cuda(), x_out=xo, raw=raw, h1=h1, h2=h2, state=state.cuda(), carry=carry, commit=prev_carry.cuda(),
                             commit_state=old)
        assert (xo.double().cpu() - total).abs().max() < 1e-5
        assert (raw.double().cpu() - total).abs().max() < tol
        assert (h1.double().cpu() - want1).abs().max() < tol
        assert (h2.double().cpu() - n * w2.double()).abs().max() < tol
        assert (carry.double().cpu() - n[last] * w1.double()).abs().max() < 2e-5      # float whatever the operand type
        assert torch.equal(old.cpu()[slots], prev_carry) and float(old[E].abs().max()) == 0.0
    # from the embedding, without a shift; and the sum alone
    h1 = torch.empty(T, W, device="cuda")
    hy.parallel_boundary(plan, emb.cuda(), eps, w1=w1.cuda(), h1=h1)
    assert (h1.double().cpu() - O.rms(emb.double()[tok], eps) * w1.double()).abs().max() < 2e-5
    raw = torch.empty(T, W, device="cuda")
    hy.parallel_boundary(plan, emb.bfloat16().cuda(), eps, o=o.cuda(), raw=raw)
    assert (raw.double().cpu() - emb.bfloat16().double()[tok] - o.double()).abs().max() < 1e-5


@pytest.mark.parametrize("C", [1, 12, 37, 300, 1536])
def test_query_latent_norm_and_output_gate(C):
    from nanorlhf_b200.ops import hybrid as hy
    g = torch.Generator().manual_seed(C)
    T, P = 9, (C + 7) // 8 * 8
    x, z = torch.randn(T, P + 8, generator=g) * 3, torch.randn(T, P + 8, generator=g) * 2
    w = torch.rand(C, generator=g) + 0.5
    for hd, tol in ((torch.float32, 1e-5), (torch.bfloat16, 5e-2)):
        out = torch.zeros(T, P, device="cuda", dtype=hd)
        hy.rmsnorm_cols(x.cuda()[:, 8:8 + C], w.cuda(), 1e-5, out[:, :C])
        assert (out.double().cpu()[:, :C] - O.rms(x.double()[:, 8:8 + C], 1e-5) * w.double()).abs().max() < tol
        out.fill_(5.0)
        hy.gate_cols(x.cuda()[:, :C], z.cuda()[:, 8:8 + C], 1.0, out[:, :C])
        assert (out.double().cpu()[:, :C] - x.double()[:, :C] * torch.sigmoid(z.double()[:, 8:8 + C])).abs().max() < tol
        assert bool((out[:, C:] == 5.0).all())


@pytest.mark.parametrize("E,top,ff", [(1, 1, 8), (5, 2, 12), (4, 4, 7), (40, 6, 32), (300, 3, 4)])
def test_sigmoid_routing_and_experts_that_read_the_weighted_input(E, top, ff):
    """Choice and weights; the dense form's activations; the grouped form (fused and plain SwiGLU) against the oracle's experts."""
    from nanorlhf_b200.ops import hybrid as hy
    g = torch.Generator().manual_seed(E * 7 + top)
    T, W = 50, 64
    h = torch.randn(T, W, generator=g).bfloat16()
    w = {"router": torch.randn(E, W, generator=g).bfloat16().double() / 8}
    mlp = dict(router=dict(experts=E, top=top))
    z = (h.double() @ w["router"].T).float()
    want_ids, want_w = O.route(w, "", mlp, h.double())
    ids, wts = torch.empty(T, top, dtype=torch.int32, device="cuda"), torch.empty(T, top, device="cuda")
    gu = torch.randn(T, E * 2 * ff, generator=g)
    act = torch.empty(T, E * ff, device="cuda")
    hy.moe_route(z.cuda(), None, top, gu=gu.cuda(), ff=ff, act=act, ids=ids, wts=wts, sigmoid=True, weight_input=True)
    assert torch.equal(ids.cpu().long(), want_ids)
    assert (wts.double().cpu() - want_w).abs().max() < 1e-6
    full = torch.zeros(T, E, dtype=torch.float64).scatter(1, want_ids, want_w)[:, :, None]
    d = gu.double().reshape(T, E, 2, ff)
    assert (act.double().cpu().reshape(T, E, ff) - O.silu(full * d[:, :, 0]) * (full * d[:, :, 1])).abs().max() < 1e-5
    if E > 40:
        return
    for F in (64, 40):                                       # 64: SwiGLU in the GEMM's epilogue; 40: a launch of its own
        for e in range(E):
            for n, (r, c) in (("gate", (F, W)), ("up", (F, W)), ("down", (W, F))):
                w[f"e{e}.{n}"] = (torch.randn(r, c, generator=g) / c ** 0.5).bfloat16()
        cat = [(hy.interleave_gate_up(w[f"e{e}.gate"], w[f"e{e}.up"]) if F % 32 == 0 else torch.cat([w[f"e{e}.gate"], w[f"e{e}.up"]])) for e in range(E)]
        wg = torch.cat(cat).cuda().contiguous()
        wd = torch.cat([w[f"e{e}.down"] for e in range(E)]).cuda().contiguous()
        y, slot_of = hy.moe_grouped_ffn(h.cuda(), ids, wts, wg, wd, E, F, None, fused_act=F % 32 == 0, weight_input=True)
        got = y[slot_of.long()].double().cpu().reshape(T, top, W).sum(1)
        want = O.moe({k: v.double() for k, v in w.items()}, "", mlp, h.double())
        assert (got - want).abs().max() < 3e-2 * want.abs().max() and (got - want).pow(2).mean().sqrt() < 1.6e-2 * want.pow(2).mean().sqrt()


def _latent_case(tmp_path, dtype, T, needles, seed=0, gain=4.0, sink=None, **sizes):
    """One latent-attention mixer driven with hand-made projections.  The query projection is ``gain`` times the identity, so that a
    query points where its latent does.  ``needles``: (query position, key position) pairs; the query is turned to head 0's
    unrotated key there, so that this one score stands far above all others (when the key is visible)."""
    H, dn, dr = sizes["heads"], sizes["dim"], sizes["rot_dim"]
    nq = H * (dn + dr)
    cfg = O.make_config(ffs=(None,), loop=None, att=dict(sizes, q_rank=nq))
    W = O.random_weights(cfg, seed=seed)
    W["l0.mix.uq"], W["l0.mix.dq.norm"] = (gain * torch.eye(nq)).bfloat16(), torch.ones(nq).bfloat16()
    if sink is not None:
        W["l0.mix.sink"] = torch.full_like(W["l0.mix.sink"], sink)
    m, r, eps = cfg["layers"][0]["mixer"], sizes["kv_rank"], cfg["norm"]["eps"]
    g = torch.Generator().manual_seed(seed + 1)
    cq = torch.randn(T, nq, generator=g, dtype=torch.float64)
    dkv = torch.randn(T, r + dr, generator=g, dtype=torch.float64)
    gate = torch.randn(T, H * sizes["vdim"], generator=g, dtype=torch.float64)
    Wd = {k: v.double() for k, v in W.items()}
    for qi, kj in needles:
        c = O.rms(dkv[kj:kj + 1, :r], eps) * Wd["l0.mix.dkv.norm"]
        cq[qi] = 0.0
        cq[qi, :dn] = (c @ Wd["l0.mix.uk"].T)[0, :dn]
    q = O.rms(cq, eps) @ Wd["l0.mix.uq"].T
    want = O.latent_core(q, dkv, Wd, "l0.mix.", m, eps) * torch.sigmoid(gate)

    def run(cuts, pool=1024):
        eng = _engine(tmp_path, cfg, W, dtype=dtype, pool_tokens=pool)
        M = eng.layers[0].mixers[0]
        sid = eng.open()
        outs, lo = [], 0
        for n in cuts:
            U = torch.zeros(n, eng.layers[0].n_in, device="cuda")
            for (c0, w), src in ((M.cols["dq"], cq), (M.cols["dkv"], dkv), (M.cols["g"], gate)):
                U[:, c0:c0 + w] = src[lo:lo + n].float().cuda()
            out = torch.empty(n, H * sizes["vdim"], device="cuda", dtype=eng.wdtype)
            eng._latent_attention(M, U, _plan(eng, [sid], [n]), eps, out)
            outs.append(out.double().cpu())
            lo += n
        eng.close(sid)
        return torch.cat(outs)
    return run, want


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
def test_latent_attention_sees_exactly_the_causal_keys(tmp_path, dtype):
    """Loud keys planted far away, at page borders, at the query's own position (the last key it sees) and one position later (the
    first it does not), in whole prompts, in portions and in single-token steps."""
    T = 330
    needles = [(300, 2), (47, 47), (15, 16), (17, 17), (31, 32), (200, 15), (255, 256), (320, 319), (329, 1), (100, 101)]
    sizes = dict(heads=3, dim=8, rot_dim=8, vdim=16, kv_rank=24, scale=0.5, base=100.0)
    run, want = _latent_case(tmp_path, dtype, T, needles, **sizes)
    tol, scale = (1e-4 if dtype == "fp32" else 4e-2), want.abs().max()
    for cuts in ([T], _cuts(T, [16, 1, 31, 2, 17]), [290] + [1] * 40):
        assert (run(cuts) - want).abs().max() < tol * scale, cuts[:4]
    # the planted keys matter: moved by one position they give another result
    _, off = _latent_case(tmp_path, dtype, T, [(q, k - 1) for q, k in needles if 0 < k <= q], **sizes)
    assert all((want[q, :16] - off[q, :16]).abs().max() > 0.1 * scale for q, k in needles if 0 < k <= q)


@pytest.mark.parametrize("sizes", [dict(heads=1, dim=4, rot_dim=4, vdim=4, kv_rank=4), dict(heads=7, dim=24, rot_dim=16, vdim=72, kv_rank=136),
                                   dict(heads=5, dim=10, rot_dim=6, vdim=14, kv_rank=20), dict(heads=20, dim=16, rot_dim=8, vdim=16, kv_rank=264),
                                   dict(heads=3, dim=16, rot_dim=64, vdim=24, kv_rank=512), dict(heads=3, dim=8, rot_dim=2, vdim=9, kv_rank=31)])
@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
def test_latent_attention_sizes(tmp_path, sizes, dtype):
    """Head counts and sizes on and off every kernel's tile, also a value size that is no multiple of the vector width."""
    run, want = _latent_case(tmp_path, dtype, 150, [(140, 3), (63, 63), (64, 63), (17, 18), (149, 16)], scale=0.2, base=1000.0, gain=2.0, **sizes)
    for cuts in ([150], [120] + [1] * 30, _cuts(150, [2, 29, 1])):
        err = (run(cuts) - want).abs().max() / want.abs().max()
        assert err < (1e-4 if dtype == "fp32" else 4e-2), cuts[:3]


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
def test_sink_counts_once_and_is_not_scaled(tmp_path, dtype):
    """A sink that takes most of the mass while few keys are seen, in prompts, portions and decoding."""
    sizes = dict(heads=2, dim=8, rot_dim=8, vdim=8, kv_rank=16, scale=0.1, base=100.0)
    run, want = _latent_case(tmp_path, dtype, 60, [], sink=3.0, gain=1.0, **sizes)
    _, none = _latent_case(tmp_path, dtype, 60, [], sink=-60.0, gain=1.0, **sizes)
    assert want[0].abs().max() < 0.1 * none[0].abs().max() and (want - none).abs().max() > 0.3 * none.abs().max()
    for cuts in ([60], [20] + [1] * 40, [2] * 30):
        assert (run(cuts) - want).abs().max() < (1e-4 if dtype == "fp32" else 3e-2) * want.abs().max()


def test_shift_alone_decides_what_the_mixer_reads(tmp_path):
    """With shift 1 the mixer sees the previous token only: the last token of a sequence cannot reach its own mixer.  In portions the
    previous row comes from the slot, and a new sequence in a used slot starts from zeros."""
    cfg = O.make_config(ffs=(None, "dense"), loop=(0, 2, 2))
    W = O.random_weights(cfg, seed=3)
    for k in W:
        if k.endswith("shift"):
            W[k] = torch.ones_like(W[k])
    eng = _engine(tmp_path, cfg, W, slots=1)
    for seed in (1, 2, 3):                                  # one slot: every sequence follows another one's state
        toks = _tokens(cfg, 40, seed)
        want = O.forward(W, cfg, toks)
        for cuts in ([40], [1] * 40, [2] * 20, _cuts(40, [16, 1, 15, 3])):
            assert _rel(_run_alone(eng, toks, cuts), want) < F32_TOL, cuts[:3]
    unshifted = {k: torch.zeros_like(v) if k.endswith("shift") else v for k, v in W.items()}
    assert _rel(O.forward(unshifted, cfg, toks), want) > 0.1


@pytest.mark.parametrize("loop", [None, (0, 1, 1), (0, 3, 2), (1, 2, 4), (1, 3, 3), (2, 3, 2)])
def test_loop_passes_and_the_stream_after_every_layer_run(tmp_path, loop):
    """Where the loop starts and stops, how often it runs, and that every pass reads pages and shifted rows of its own."""
    cfg = O.make_config(ffs=("dense", "moe", None), loop=loop)
    W = O.random_weights(cfg, seed=2)
    toks = _tokens(cfg, 33, 2)
    keep_want = []
    want = O.forward(W, cfg, toks, keep=keep_want)
    eng = _engine(tmp_path, cfg, W)
    sid = eng.open()
    got = []
    for lo, hi in ((0, 19), (19, 20), (20, 33)):
        keep = []
        eng._forward_parallel(_plan(eng, [sid], [hi - lo], toks[lo:hi]), [], keep)
        got.append(keep)
    assert all(len(k) == len(keep_want) == len(O.schedule(cfg)) for k in got)
    for i, ref in enumerate(keep_want):
        x = torch.cat([k[i] for k in got]).double().cpu()
        assert (x - ref).abs().max() < 1e-4 * ref.abs().max(), i
    eng.close(sid)
    assert _rel(_run_alone(eng, toks, _cuts(33, [7, 1, 2])), want) < F32_TOL
    if loop and loop[2] > 1:                                # weights are shared by the passes, pages and state are not
        runs = [L for L in eng.layers if L.spec.index == loop[0]]
        assert len(runs) == loop[2] and len({L.w_in.data_ptr() for L in runs}) == 1
        assert len({L.mixers[0].k_cache.data_ptr() for L in runs}) == len({L.shift_state.data_ptr() for L in runs}) == loop[2]


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
    """One- and two-token sequences: position 0 (no rotation, zeros in front of the shift), a sink beside a single key."""
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
    """Hundreds of single-token steps: the shifted row is carried and the attention keeps every key."""
    cfg, W = _model("odd")
    toks = _tokens(cfg, 260, 8)
    eng = _engine(tmp_path, cfg, W)
    assert _rel(_run_alone(eng, toks, [4] + [1] * 256), O.forward(W, cfg, toks)) < F32_TOL


def test_distant_tokens_reach_through_the_cache(tmp_path):
    """Changing an early token must change late logits, in the engine as in the oracle, in portions and in decoding."""
    cfg = O.make_config(ffs=("dense", None), loop=(0, 1, 2))
    W = O.random_weights(cfg, seed=4)
    a = _tokens(cfg, 150, 3)
    b = list(a)
    b[1] = (b[1] + 1) % cfg["vocab"]
    wa, wb = O.forward(W, cfg, a), O.forward(W, cfg, b)
    assert _rel(wa[-8:], wb[-8:]) > 10 * F32_TOL
    eng = _engine(tmp_path, cfg, W)
    for toks, want in ((a, wa), (b, wb)):
        assert _rel(_run_alone(eng, toks, [130] + [1] * 20)[-8:], want[-8:]) < F32_TOL


def test_grouped_and_dense_expert_forms_agree(tmp_path):
    """bf16 serving runs only the chosen experts (rows sorted by expert, the sums formed in the next boundary); the dense form runs
    every expert.  Both against the oracle, with the SwiGLU in the GEMM's epilogue and as a launch of its own."""
    for ff in (32, 24):
        cfg = O.make_config(ffs=("moe", "moe"), width=64, loop=(1, 2, 2), moe=dict(ff=ff, experts=6, top=3))
        W = _decisive_routers(O.random_weights(cfg, seed=9))
        toks = _tokens(cfg, 150, 4)
        want = O.forward(W, cfg, toks)
        for form in ("grouped", "dense"):
            eng = _engine(tmp_path, cfg, W, dtype="bf16", name=form, moe=form)
            assert any(L.ff.w_gate_up is not None for L in eng.layers) == (form == "grouped")
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
    """``python -m nanorlhf_b200.sampler`` on a Lopovik checkpoint: the class and the engine come from config.json."""
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
