"""Plain float64 implementation of the Lopovik decoder, one function per mechanism, written from the design's equations.

It shares no code with the serving path: whole sequences only, no cache, no pages, no batching; the token shift looks at the
row above, keys and values are expanded per head and every attention builds its full score matrix.  ``weights`` maps checkpoint
tensor names to tensors, ``cfg`` is the parsed ``config.json``.
"""
import math

import torch

F64 = torch.float64


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def centred_norm(x, weight, eps):
    """RMS norm whose weight is stored around zero."""
    return rms(x, eps) * (1.0 + weight)


def silu(z):
    return z * torch.sigmoid(z)


def token_shift(h, mu):
    """Every row moves towards the row of the previous token, per column by ``mu``; in front of the first token are zeros."""
    prev = torch.cat([torch.zeros_like(h[:1]), h[:-1]], 0)
    return h + (prev - h) * mu


def rotate_pairs(x, positions, rot):
    """x [tokens, ..., n]: columns 2i and 2i + 1 of the first ``dims`` turn by position * base^(-2i / dims); the others pass."""
    dims, base = int(rot["dims"]), float(rot["base"])
    f = base ** (-2.0 * torch.arange(dims // 2, dtype=F64) / dims)
    a = positions.to(F64)[:, None] * f[None, :]
    a = a.reshape([x.shape[0]] + [1] * (x.dim() - 2) + [dims // 2])
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * torch.cos(a) - v * torch.sin(a)
    out[..., 1:dims:2] = v * torch.cos(a) + u * torch.sin(a)
    return out


def query_latent(w, p, h, eps):
    """Queries of all heads [T, H * (dim + rot_dim)] through a normed low-rank latent."""
    return (rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]) @ w[p + "uq"].T


def latent_core(q, dkv, w, p, m, eps, positions=None):
    """Attention from the projections: q [T, H * (dim + rot_dim)], dkv [T, kv_rank + rot_dim] -> heads [T, H * vdim], not gated."""
    T = q.shape[0]
    H, dn, dr, dv, r = int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"])
    pos = torch.arange(T) if positions is None else positions
    q = q.reshape(T, H, dn + dr)
    qn, qr = q[..., :dn], rotate_pairs(q[..., dn:], pos, m["rot"])
    c = rms(dkv[:, :r], eps) * w[p + "dkv.norm"]
    kr = rotate_pairs(dkv[:, r:], pos, m["rot"])
    kn = (c @ w[p + "uk"].T).reshape(T, H, dn)
    v = (c @ w[p + "uv"].T).reshape(T, H, dv)
    out = torch.zeros(T, H, dv, dtype=F64)
    mask = torch.tril(torch.ones(T, T, dtype=torch.bool))
    for hd in range(H):
        s = (qn[:, hd] @ kn[:, hd].T + qr[:, hd] @ kr.T) * float(m["scale"])
        out[:, hd] = sink_softmax(s.masked_fill(~mask, -math.inf), w[p + "sink"][hd]) @ v[:, hd]
    return out.reshape(T, H * dv)


def sink_softmax(s, sink):
    """Softmax over the last axis whose denominator holds exp(sink) once more."""
    mx = torch.maximum(s.max(-1, keepdim=True).values, sink)
    e = torch.exp(s - mx)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - mx))


def latent_attention(w, p, m, h, eps):
    heads = latent_core(query_latent(w, p, h, eps), h @ w[p + "dkv"].T, w, p, m, eps)
    return (heads * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def relu2_ff(w, p, h):
    return torch.relu(h @ w[p + "up"].T) ** 2 @ w[p + "down"].T


def expert(w, p, h):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(w, p, mlp, h):
    """Chosen experts [T, top] and their weights, the sigmoid scores themselves."""
    s = torch.sigmoid(h @ w[p + "router"].T)
    ws, ids = torch.topk(s, int(mlp["router"]["top"]), dim=-1)
    return ids, ws


def moe(w, p, mlp, h):
    """Every chosen expert reads the input times its score; the results are summed as they are."""
    ids, ws = route(w, p, mlp, h)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, a in zip(ids[t].tolist(), ws[t]):
            out[t] += expert(w, f"{p}e{e}.", a * h[t:t + 1])[0]
    return out


def feed_forward(w, p, mlp, h):
    return relu2_ff(w, p, h) if mlp["kind"] == "dense" else moe(w, p, mlp, h)


def layer(w, cfg, i, x, eps):
    """Mixer and feed-forward side by side on the same x, each behind its own norm; only the mixer's input is shifted."""
    p, spec = f"l{i}.", cfg["layers"][i]
    h = token_shift(centred_norm(x, w[p + "norm1"], eps), w[p + "shift"])
    y = latent_attention(w, p + "mix.", spec["mixer"], h, eps)
    if spec.get("mlp"):
        y = y + feed_forward(w, p + "mlp.", spec["mlp"], centred_norm(x, w[p + "norm2"], eps))
    return x + y


def pass_entry(w, x, x0):
    return torch.cat([x, x0], -1) @ w["loop.in"].T


def schedule(cfg):
    """(layer index, is the first layer of a pass of the loop) in the order of execution."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = int(loop["start"]), int(loop["stop"])
    out = [(i, False) for i in range(a)]
    for _ in range(int(loop["times"])):
        out += [(i, i == a) for i in range(a, b)]
    return out + [(i, False) for i in range(b, n)]


def forward(weights, cfg, tokens, keep=None):
    """Logits [tokens, vocab] of one whole sequence; ``keep`` receives the stream after every layer that was run."""
    w = {k: v.to(F64) if v.is_floating_point() else v for k, v in weights.items()}
    eps = float(cfg["norm"]["eps"])
    x0 = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    x = x0
    for i, entry in schedule(cfg):
        if entry:
            x = pass_entry(w, x, x0)
        x = layer(w, cfg, i, x, eps)
        if keep is not None:
            keep.append(x.clone())
    return centred_norm(x, w["final.norm"], eps) @ w["embed"].T


# ---- small configurations and random weights for the tests ------------------------------------------------------------
def make_config(vocab=97, width=48, eps=1e-5, ffs=("dense", "moe", None), att=None, dense_ff=40, moe=None, loop=(1, 2, 2), per_layer=None):
    """A ``config.json`` dictionary.  ``ffs``: per layer "dense" | "moe" | None; ``loop``: (start, stop, times) or None; ``per_layer``:
    {layer index: overrides of the mixer's sizes}."""
    a = dict(heads=3, dim=8, rot_dim=4, vdim=10, kv_rank=16, q_rank=20, scale=0.3, base=10000.0)
    a.update(att or {})
    mo = dict(ff=16, experts=5, top=2)
    mo.update(moe or {})
    layers = []
    for i, kind in enumerate(ffs):
        s = dict(a, **(per_layer or {}).get(i, {}))
        mixer = {k: s[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank", "scale")}
        mixer["rot"] = dict(base=s["base"], dims=s["rot_dim"])
        mlp = None
        if kind == "dense":
            mlp = dict(kind="dense", ff=dense_ff)
        elif kind == "moe":
            mlp = dict(kind="moe", expert=dict(ff=mo["ff"]), router=dict(experts=mo["experts"], top=mo["top"]))
        layers.append(dict(type="latent_attention", mixer=mixer, mlp=mlp))
    cfg = dict(architecture="Lopovik", vocab=vocab, width=width, norm=dict(eps=eps), layers=layers)
    if loop:
        cfg["loop"] = dict(start=loop[0], stop=loop[1], times=loop[2])
    return cfg


def random_weights(cfg, seed=0, dtype=torch.bfloat16):
    """Random checkpoint tensors for ``cfg`` (rounded to ``dtype``, so that the oracle and the engine read the same numbers)."""
    gen = torch.Generator().manual_seed(seed)
    W = cfg["width"]
    w = {}

    def lin(name, o, i, s=1.0):
        w[name] = torch.randn(o, i, generator=gen) * s / i ** 0.5
    w["embed"] = torch.randn(cfg["vocab"], W, generator=gen)
    if cfg.get("loop"):
        lin("loop.in", W, 2 * W)
    for i, spec in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", spec["mixer"], spec.get("mlp")
        w[p + "norm1"] = torch.randn(W, generator=gen) * 0.2
        w[p + "shift"] = torch.rand(W, generator=gen)
        q, H, r = p + "mix.", m["heads"], m["kv_rank"]
        lin(q + "dq", m["q_rank"], W), lin(q + "uq", H * (m["dim"] + m["rot_dim"]), m["q_rank"])
        lin(q + "dkv", r + m["rot_dim"], W)
        w[q + "dq.norm"], w[q + "dkv.norm"] = torch.rand(m["q_rank"], generator=gen) + 0.5, torch.rand(r, generator=gen) + 0.5
        lin(q + "uk", H * m["dim"], r), lin(q + "uv", H * m["vdim"], r)
        w[q + "sink"] = torch.randn(H, generator=gen)
        lin(q + "g", H * m["vdim"], W), lin(q + "o", W, H * m["vdim"])
        f = p + "mlp."
        if mlp is None:
            continue
        w[p + "norm2"] = torch.randn(W, generator=gen) * 0.2
        if mlp["kind"] == "dense":
            lin(f + "up", mlp["ff"], W), lin(f + "down", W, mlp["ff"])
        else:
            ff = mlp["expert"]["ff"]
            for e in range(mlp["router"]["experts"]):
                lin(f"{f}e{e}.gate", ff, W, 1.5), lin(f"{f}e{e}.up", ff, W), lin(f"{f}e{e}.down", W, ff)
            lin(f + "router", mlp["router"]["experts"], W)
    w["final.norm"] = torch.randn(W, generator=gen) * 0.2
    return {k: v.to(dtype) for k, v in w.items()}
