"""CPU-side checks of the Lapilorn family: registry, configuration, tensor inventory, checkpoint round trip, host tables, and the
oracle's own invariants (the GPU tests compare the engine with this oracle)."""
import json
import math
import os

import pytest
import torch

import lapilorn_oracle as O


def _save(tmp_path, cfg, W, name="m"):
    from safetensors.torch import save_file
    d = os.path.join(str(tmp_path), name)
    os.makedirs(d, exist_ok=True)
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in W.items()}, os.path.join(d, "model.safetensors"))
    return d


LAYERS = ("attention/dense", "lightning/moe", "attention/moe", "lightning/dense", "attention/none", "lightning/none")


def test_registry_resolves_by_architecture():
    from nanorlhf_b200.models.lapilorn import LapilornForCausalLM
    from nanorlhf_b200.models.registry import resolve
    cls, kind = resolve({"architecture": "Lapilorn"})
    assert cls is LapilornForCausalLM and kind == "hybrid"
    assert resolve({"model_type": "lapilorn"})[0] is LapilornForCausalLM


def test_config_reads_every_size_and_constant():
    from nanorlhf_b200.models.lapilorn import LapilornConfig
    rot = dict(base=777.0, dims=6, scaling=dict(factor=3.0, low=0.5, high=9.0, original=100))
    d = O.make_config(vocab=211, width=56, eps=3e-4, layers=LAYERS, kv_from={4: 2}, ff=72, limit=2.5,
                      att=dict(heads=6, kv_heads=2, dim=10, vdim=14, scale=0.77, softcap=11.0, rot=rot),
                      lin=dict(heads=2, dim=20, vdim=6, decay=[0.25, 0.875]), per_layer={0: dict(heads=3, kv_heads=3, dim=4, vdim=30, rot=None)},
                      moe=dict(ff=24, experts=12, top=4, scale=0.6, groups=dict(count=4, keep=3), shared=40))
    c = LapilornConfig.from_dict(d)
    st, specs = c.stream_spec(), c.layer_specs()
    assert (st.kind, st.shared_norm, st.centred_norm, st.token_shift, st.loop, st.tied_head, st.positions) == ("parallel", True, True, False, None, True, False)
    assert c.norm_eps == 3e-4 and (c.vocab_size, c.hidden_size, c.num_hidden_layers) == (211, 56, 6)
    a, b, li = specs[2].mixers[0], specs[0].mixers[0], specs[1].mixers[0]
    assert (a.kind, a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.softcap, a.rot_dims, a.rot_base, a.rot_layout, a.rot_scaling, a.kv_from) == \
        ("rot_attention", 6, 2, 10, 14, 0.77, 11.0, 6, 777.0, "interleaved", rot["scaling"], -1)
    assert a.out_gate and a.window == 0 and a.maps == 1 and not a.qk_bias and not a.head_sink and not a.unit_qk_norm
    assert (b.heads, b.kv_heads, b.dim, b.vdim, b.rot_dims) == (3, 3, 4, 30, 0) and specs[4].mixers[0].kv_from == 2
    assert (li.kind, li.heads, li.dim, li.vdim, li.decay, li.norm_groups) == ("lightning", 2, 20, 6, (0.25, 0.875), 1)
    m, f = specs[1], specs[0]
    assert (m.ff, m.ff_kind, m.ff_act, m.experts, m.top, m.route, m.route_scale, m.route_groups, m.route_keep, m.group_score, m.shared_ff) == \
        (24, "moe", "relu2", 12, 4, "sigmoid_all", 0.6, 4, 3, "top2", 40)
    assert (f.ff, f.ff_kind, f.ff_act, f.ff_limit, f.ff_alpha, f.ff_up_shift) == (72, "dense", "swiglu", 2.5, 1.702, 1.0)
    assert specs[4].ff == 0 and specs[5].ff == 0
    assert LapilornConfig.from_dict(c.to_dict()).to_dict() == c.to_dict()
    # no scaling, no groups, no shared expert
    p = O.make_config(att=dict(rot=dict(base=50.0, dims=4)), moe=dict(groups=None, shared=None))
    s = LapilornConfig.from_dict(p).layer_specs()
    assert s[0].mixers[0].rot_scaling is None and s[1].route_groups == 1 and s[1].shared_ff == 0


def test_what_the_engine_cannot_run_is_refused():
    from nanorlhf_b200.models.lapilorn import LapilornConfig

    def refused(change):
        d = json.loads(json.dumps(O.make_config(layers=LAYERS)))
        change(d["layers"])
        with pytest.raises(ValueError):
            LapilornConfig.from_dict(d)
    refused(lambda ls: ls[0].update(type="ssm"))
    refused(lambda ls: ls[0]["mlp"].update(kind="glu"))
    refused(lambda ls: ls[0]["mlp"].update(limit=0.0))
    refused(lambda ls: ls[0]["mixer"].update(kv_heads=3))
    refused(lambda ls: ls[0]["mixer"]["rot"].update(dims=7))
    refused(lambda ls: ls[0]["mixer"]["rot"].update(dims=14))
    refused(lambda ls: ls[1]["mixer"].update(decay=[0.5]))
    refused(lambda ls: ls[2]["mixer"].update(kv_from=2))                # itself
    refused(lambda ls: ls[2]["mixer"].update(kv_from=4))                # a later layer
    refused(lambda ls: ls[2]["mixer"].update(kv_from=1))                # a layer of another kind
    refused(lambda ls: (ls[2]["mixer"].update(kv_from=0), ls[4]["mixer"].update(kv_from=2)))     # a layer that borrows itself
    refused(lambda ls: ls[2]["mixer"].update(kv_from=0, vdim=12))
    refused(lambda ls: ls[1]["mlp"]["router"].update(top=7))
    refused(lambda ls: ls[1]["mlp"]["router"].update(groups=dict(count=4, keep=2)))
    refused(lambda ls: ls[1]["mlp"]["router"].update(groups=dict(count=3, keep=4)))
    refused(lambda ls: ls[1]["mlp"]["router"].update(top=3, groups=dict(count=3, keep=1)))


def test_tensor_inventory_matches_the_oracle_weights_and_round_trips(tmp_path):
    from nanorlhf_b200.models.lapilorn import LapilornConfig
    from nanorlhf_b200.models.registry import load_model
    d = O.make_config(layers=LAYERS, kv_from={4: 0})
    W = O.random_weights(d, seed=1)
    shapes = LapilornConfig.from_dict(d).tensor_shapes()
    assert set(shapes) == set(W) and all(tuple(W[n].shape) == tuple(s) for n, s in shapes.items())
    assert "l4.mix.k" not in shapes and "l4.mix.v" not in shapes and "l5.mlp.up" not in shapes
    m = load_model(_save(tmp_path, d, W), torch_dtype=torch.bfloat16)
    assert all(torch.equal(m.tensor(n), W[n]) for n in W)
    m.save_pretrained(os.path.join(str(tmp_path), "again"))
    m2 = load_model(os.path.join(str(tmp_path), "again"))
    assert all(torch.equal(m.tensor(n), m2.tensor(n)) for n in m.names)
    for change in (lambda w: w.update({"l0.mix.k": w["l0.mix.k"][:-1].contiguous()}), lambda w: w.pop("l1.mix.norm"), lambda w: w.pop("l1.mlp.correction"),
                   lambda w: w.pop("l3.mlp.gate"), lambda w: w.pop("l2.mlp.shared.up")):
        bad = dict(W)
        change(bad)
        with pytest.raises(ValueError):
            load_model(_save(tmp_path, d, bad, "bad"))


def test_random_init_from_config():
    from nanorlhf_b200.models.lapilorn import LapilornConfig, LapilornForCausalLM
    m = LapilornForCausalLM.from_config(LapilornConfig.from_dict(O.make_config(layers=LAYERS)), seed=3)
    assert all(torch.isfinite(m.tensor(n).float()).all() for n in m.names)


@pytest.mark.parametrize("dims,base,sc", [(16, 1e4, dict(factor=8.0, low=1.0, high=4.0, original=256)), (8, 50.0, dict(factor=3.0, low=0.25, high=2.0, original=37)),
                                          (64, 5e5, dict(factor=16.0, low=1.0, high=4.0, original=8192)), (2, 10.0, dict(factor=2.0, low=1.0, high=4.0, original=3)),
                                          (12, 1e3, None)])
def test_frequency_table(dims, base, sc):
    from nanorlhf_b200.ops.hybrid import rotary_frequencies
    f, mult = rotary_frequencies(dims, base, sc)
    want = O.frequencies(dict(dims=dims, base=base, scaling=sc))
    assert mult == 1.0 and torch.allclose(torch.tensor(f, dtype=torch.float64), want, rtol=1e-14, atol=0)
    if sc:                                                   # by wavelength, as the scaling is defined
        for i, x in enumerate(f):
            raw = base ** (-2.0 * i / dims)
            wave = 2 * math.pi / raw
            if wave < sc["original"] / sc["high"]:
                assert x == raw
            elif wave > sc["original"] / sc["low"]:
                assert abs(x - raw / sc["factor"]) < 1e-15 * raw
            else:
                assert raw / sc["factor"] * (1 - 1e-12) <= x <= raw * (1 + 1e-12)


def test_decay_powers_are_exact():
    from nanorlhf_b200.ops.hybrid import LIGHTNING_CHUNK, decay_powers
    p = decay_powers([0.0, 0.25, 1.0, 0.9990234375], "cpu")
    assert p.shape == (4, LIGHTNING_CHUNK + 1) and p.dtype == torch.float32
    assert p[0].tolist() == [1.0] + [0.0] * LIGHTNING_CHUNK and bool((p[2] == 1).all()) and p[1, 10] == 0.25 ** 10
    assert abs(float(p[3, -1]) / 0.9990234375 ** LIGHTNING_CHUNK - 1) < 1e-7


# ---- the oracle's own invariants -------------------------------------------------------------------------------------
def test_oracle_is_causal_and_borrowed_keys_are_the_other_layers():
    d = O.make_config(layers=LAYERS, kv_from={4: 0})
    W = O.random_weights(d, seed=5)
    toks = [1, 2, 3, 4, 5, 6, 7, 8, 9, 10, 11]
    full, keep = O.forward(W, d, toks), []
    assert (O.forward(W, d, toks[:6], keep) - full[:6]).abs().max() < 1e-9 and len(keep) == 6
    # projections of its own that give the same keys and values would need the other layer's input
    W2 = dict(W, **{"l4.mix.k": W["l0.mix.k"], "l4.mix.v": W["l0.mix.v"]})
    assert (O.forward(W2, O.make_config(layers=LAYERS), toks) - full).abs().max() > 1e-2


def test_oracle_linear_attention_equals_its_expanded_sum():
    g = torch.Generator().manual_seed(3)
    q, k, v = (torch.randn(9, 2, n, generator=g, dtype=torch.float64) for n in (4, 4, 3))
    decay = [0.5, 0.99]
    o, S = O.lightning_core(q, k, v, decay)
    for h in range(2):
        for t in range(9):
            want = sum(decay[h] ** (t - j) * (q[t, h] @ k[j, h]) * v[j, h] for j in range(t + 1))
            assert (o[t, h] - want).abs().max() < 1e-12
    o1, S1 = O.lightning_core(q[:4], k[:4], v[:4], decay)
    o2, S2 = O.lightning_core(q[4:], k[4:], v[4:], decay, S1)
    assert (torch.cat([o1, o2]) - o).abs().max() < 1e-12 and (S2 - S).abs().max() < 1e-12


def test_oracle_cap_rotation_and_clamp():
    s = torch.tensor([-1e4, -1.0, 0.0, 1e-3, 1e4], dtype=torch.float64)
    c = O.cap(s, 5.0)
    assert abs(float(c[4]) - 5.0) < 1e-9 and abs(float(c[0]) + 5.0) < 1e-9 and abs(float(c[3]) - 1e-3) < 1e-9 and torch.equal(O.cap(s, 0.0), s)
    x, y = torch.randn(1, 1, 8, dtype=torch.float64), torch.randn(1, 1, 8, dtype=torch.float64)
    rot = dict(base=100.0, dims=6, scaling=dict(factor=4.0, low=1.0, high=4.0, original=50))

    def score(pq, pk):
        return float((O.rotate_pairs(x, torch.tensor([pq]), rot) * O.rotate_pairs(y, torch.tensor([pk]), rot)).sum())
    assert abs(score(9, 4) - score(105, 100)) < 1e-9 and abs(score(9, 4) - score(9, 5)) > 1e-6
    one = torch.tensor([5.0, -5.0, 0.5], dtype=torch.float64)
    got = O.clamped_glu(one, -one, 2.0)
    want = [2 / (1 + math.exp(-3.404)) * -1.0, -5 / (1 + math.exp(8.51)) * 3.0, 0.5 / (1 + math.exp(-0.851)) * 0.5]
    assert (got - torch.tensor(want, dtype=torch.float64)).abs().max() < 1e-12


def test_oracle_router_by_hand():
    """A closed group holds a better expert than a chosen one; a group wins by its two best together; choice scores are negative; the
    weights leave the correction out."""
    z = torch.logit(torch.tensor([0.9, 0.1, 0.6, 0.5, 0.3, 0.2], dtype=torch.float64))
    corr = torch.full((6,), -1.0, dtype=torch.float64)
    r = dict(experts=6, top=2, scale=2.0, groups=dict(count=3, keep=1))
    got = O.route(z, corr, r)                                # groups: 0.9 + 0.1 < 0.6 + 0.5
    assert [e for e, _ in got] == [2, 3] and abs(got[0][1] - 2 * 0.6 / 1.1) < 1e-9 and abs(got[1][1] - 2 * 0.5 / 1.1) < 1e-9
    corr[1] += 0.2
    got = O.route(z, corr, r)                                # now 0.9 + 0.3 > 1.1; the weight of expert 1 is still its plain score
    assert [e for e, _ in got] == [0, 1] and abs(got[1][1] - 2 * 0.1 / 1.0) < 1e-9
    got = O.route(z, corr, dict(r, groups=None))
    assert [e for e, _ in got] == [0, 2]
