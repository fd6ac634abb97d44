"""CPU-side checks of the Lopovik family: registry, configuration, tensor inventory, checkpoint round trip, and the oracle's own
invariants (the GPU tests compare the engine with this oracle)."""
import json
import os

import pytest
import torch

import lopovik_oracle as O


def _save(tmp_path, cfg, W, name="m"):
    from safetensors.torch import save_file
    d = os.path.join(str(tmp_path), name)
    os.makedirs(d, exist_ok=True)
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in W.items()}, os.path.join(d, "model.safetensors"))
    return d


def test_registry_resolves_by_architecture():
    from nanorlhf_b200.models.lopovik import LopovikForCausalLM
    from nanorlhf_b200.models.registry import resolve
    cls, kind = resolve({"architecture": "Lopovik"})
    assert cls is LopovikForCausalLM and kind == "hybrid"
    assert resolve({"model_type": "lopovik"})[0] is LopovikForCausalLM


def test_config_reads_every_size_and_constant():
    from nanorlhf_b200.models.lopovik import LopovikConfig
    d = O.make_config(vocab=211, width=56, eps=3e-4, ffs=("moe", None, "dense"), dense_ff=72, loop=(0, 2, 5),
                      att=dict(heads=5, dim=12, rot_dim=6, vdim=14, kv_rank=20, q_rank=9, scale=0.77, base=777.0),
                      per_layer={2: dict(heads=2, dim=4, rot_dim=2, vdim=30, kv_rank=11, q_rank=40, scale=0.1, base=50.0)},
                      moe=dict(ff=24, experts=9, top=4))
    c = LopovikConfig.from_dict(d)
    st, specs = c.stream_spec(), c.layer_specs()
    assert (st.kind, st.token_shift, st.centred_norm, st.loop, st.tied_head, st.positions) == ("parallel", True, True, (0, 2, 5), True, False)
    assert c.norm_eps == 3e-4 and (c.vocab_size, c.hidden_size, c.num_hidden_layers) == (211, 56, 3)
    a, b = specs[0].mixers[0], specs[2].mixers[0]
    assert (a.kind, a.heads, a.kv_heads, a.dim, a.rot_dim, a.rot_dims, a.vdim, a.kv_rank, a.q_rank, a.scale, a.rot_base, a.rot_layout) == \
        ("latent_attention", 5, 1, 12, 6, 6, 14, 20, 9, 0.77, 777.0, "interleaved")
    assert a.head_sink and a.out_gate and not a.head_gate and a.rot_scaling is None
    assert (b.heads, b.dim, b.rot_dim, b.vdim, b.kv_rank, b.q_rank, b.scale, b.rot_base) == (2, 4, 2, 30, 11, 40, 0.1, 50.0)
    m = specs[0]
    assert (m.ff, m.ff_kind, m.ff_act, m.experts, m.top, m.route, m.weight_input) == (24, "moe", "swiglu", 9, 4, "sigmoid", True)
    assert specs[1].ff == 0 and (specs[2].ff, specs[2].ff_kind, specs[2].ff_act) == (72, "dense", "relu2")
    assert LopovikConfig.from_dict(c.to_dict()).to_dict() == c.to_dict()
    assert "l1.norm2" not in c.tensor_shapes() and c.tensor_shapes()["loop.in"] == (56, 112)
    c2 = LopovikConfig.from_dict(O.make_config(loop=None))
    assert c2.stream_spec().loop is None and "loop.in" not in c2.tensor_shapes() and "loop" not in c2.to_dict()


def test_what_the_engine_cannot_run_is_refused():
    from nanorlhf_b200.models.lopovik import LopovikConfig

    def refused(change):
        d = O.make_config()
        change(d)
        with pytest.raises(ValueError):
            LopovikConfig.from_dict(d)
    refused(lambda d: d["layers"][0].update(type="ssm"))
    refused(lambda d: d["layers"][0]["mlp"].update(kind="glu"))
    refused(lambda d: d["layers"][0]["mixer"]["rot"].update(dims=6))
    refused(lambda d: d["layers"][0]["mixer"]["rot"].update(dims=3))
    refused(lambda d: d["layers"][1]["mlp"]["router"].update(top=6))
    refused(lambda d: d.update(loop=dict(start=1, stop=4, times=2)))
    refused(lambda d: d.update(loop=dict(start=2, stop=2, times=2)))
    refused(lambda d: d.update(loop=dict(start=0, stop=1, times=0)))


def test_tensor_inventory_matches_the_oracle_weights_and_round_trips(tmp_path):
    from nanorlhf_b200.models.lopovik import LopovikConfig
    from nanorlhf_b200.models.registry import load_model
    d = O.make_config(ffs=("dense", "moe", None, "moe"), loop=(1, 4, 2))
    W = O.random_weights(d, seed=1)
    shapes = LopovikConfig.from_dict(d).tensor_shapes()
    assert set(shapes) == set(W) and all(tuple(W[n].shape) == tuple(s) for n, s in shapes.items())
    m = load_model(_save(tmp_path, d, W), torch_dtype=torch.bfloat16)
    assert all(torch.equal(m.tensor(n), W[n]) for n in W)
    m.save_pretrained(os.path.join(str(tmp_path), "again"))
    m2 = load_model(os.path.join(str(tmp_path), "again"))
    assert all(torch.equal(m.tensor(n), m2.tensor(n)) for n in m.names)
    extra = dict(W)
    extra["l2.norm2"] = torch.zeros(48)                             # a norm of a feed-forward the layer does not have: not read
    assert not load_model(_save(tmp_path, d, extra, "extra")).has_tensor("l2.norm2")
    for change in (lambda w: w.update({"l1.mix.uk": w["l1.mix.uk"][:-1]}), lambda w: w.pop("l1.mix.sink"), lambda w: w.pop("l3.shift"),
                   lambda w: w.update({"loop.in": w["loop.in"][:, :-1].contiguous()})):
        bad = dict(W)
        change(bad)
        with pytest.raises(ValueError):
            load_model(_save(tmp_path, d, bad, "bad"))


def test_random_init_from_config():
    from nanorlhf_b200.models.lopovik import LopovikConfig, LopovikForCausalLM
    m = LopovikForCausalLM.from_config(LopovikConfig.from_dict(O.make_config()), seed=3)
    assert all(torch.isfinite(m.tensor(n).float()).all() for n in m.names)


def test_interleaving_of_expert_rows_keeps_gate_and_up_of_a_feature_together():
    from nanorlhf_b200.ops.hybrid import interleave_gate_up
    g, u = torch.arange(64.0)[:, None], 100.0 + torch.arange(64.0)[:, None]
    z = interleave_gate_up(g, u)[:, 0].tolist()
    assert z[:32] == list(range(32)) and z[32:64] == [100.0 + i for i in range(32)] and z[64:96] == list(range(32, 64))


# ---- the oracle's own invariants -------------------------------------------------------------------------------------
def test_oracle_is_causal_and_runs_the_loop_in_order():
    d = O.make_config(ffs=("dense", "moe", None, "dense"), loop=(1, 3, 3))
    W = O.random_weights(d, seed=5)
    assert O.schedule(d) == [(0, False), (1, True), (2, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    toks = [1, 2, 3, 4, 5, 6, 7, 8, 9, 10, 11]
    full, keep = O.forward(W, d, toks), []
    assert (O.forward(W, d, toks[:6], keep) - full[:6]).abs().max() < 1e-9 and len(keep) == 8
    # a projection that passes x and drops the embedding makes a single pass a plain stack
    W["loop.in"] = torch.cat([torch.eye(48), torch.zeros(48, 48)], 1)
    once, none = O.make_config(ffs=("dense", "moe"), loop=(0, 2, 1)), O.make_config(ffs=("dense", "moe"), loop=None)
    assert (O.forward(W, once, toks) - O.forward(W, none, toks)).abs().max() < 1e-9


def test_oracle_shift_sink_and_rotation():
    h = torch.randn(6, 5, dtype=torch.float64)
    s = O.token_shift(h, torch.tensor([0.0, 1.0, 0.25, 0.0, 1.0], dtype=torch.float64))
    assert torch.equal(s[:, 0], h[:, 0]) and torch.allclose(s[1:, 1], h[:-1, 1]) and s[0, 1] == 0 and abs(float(s[0, 2] - 0.75 * h[0, 2])) < 1e-12
    x, y = torch.randn(1, 8, dtype=torch.float64), torch.randn(1, 8, dtype=torch.float64)
    rot = dict(base=100.0, dims=6)

    def score(pq, pk):
        return float((O.rotate_pairs(x, torch.tensor([pq]), rot) * O.rotate_pairs(y, torch.tensor([pk]), rot)).sum())
    assert abs(score(9, 4) - score(105, 100)) < 1e-9 and abs(score(9, 4) - score(9, 5)) > 1e-6
    p = O.sink_softmax(torch.tensor([[0.0, 1.0, float("-inf")]], dtype=torch.float64), torch.tensor(0.5, dtype=torch.float64))
    e = torch.exp(torch.tensor([0.0, 1.0, 0.5], dtype=torch.float64))
    assert torch.allclose(p[0, :2], e[:2] / e.sum()) and p[0, 2] == 0
    big = O.sink_softmax(torch.zeros(1, 3, dtype=torch.float64), torch.tensor(60.0, dtype=torch.float64))
    assert big.abs().max() < 1e-12


def test_oracle_experts_read_the_weighted_input():
    d = O.make_config(ffs=("moe",), loop=None, moe=dict(experts=2, top=2))
    W = {k: v.double() for k, v in O.random_weights(d, seed=6).items()}
    h = torch.randn(5, 48, dtype=torch.float64)
    s = torch.sigmoid(h @ W["l0.mlp.router"].T)
    want = sum(O.expert(W, f"l0.mlp.e{e}.", s[:, e:e + 1] * h) for e in range(2))
    got = O.moe(W, "l0.mlp.", d["layers"][0]["mlp"], h)
    assert (got - want).abs().max() < 1e-9
    outside = sum(s[:, e:e + 1] * O.expert(W, f"l0.mlp.e{e}.", h) for e in range(2))
    assert (got - outside).abs().max() > 1e-2                       # not the same as a weight on the result
