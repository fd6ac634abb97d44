"""Plain float64 implementation of the Lapilorn decoder, one function per mechanism, written from the design's equations.

It shares no code with the serving path: whole sequences only, no cache, no pages, no batching; every attention builds its full
score matrix and the linear attention is a loop over tokens.  ``weights`` maps checkpoint tensor names to tensors, ``cfg`` is the
parsed ``config.json``.
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


def frequencies(rot):
    """One frequency per rotated pair; long wavelengths are stretched by ``factor``, those in the middle band blended."""
    dims, base, sc = int(rot["dims"]), float(rot["base"]), rot.get("scaling")
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if sc:
            turns = float(sc["original"]) * f / (2.0 * math.pi)      # how often the pair turns within the original length
            if turns < float(sc["low"]):
                f = f / float(sc["factor"])
            elif turns <= float(sc["high"]):
                s = (turns - float(sc["low"])) / (float(sc["high"]) - float(sc["low"]))
                f = (1.0 - s) * f / float(sc["factor"]) + s * f
        out.append(f)
    return torch.tensor(out, dtype=F64)


def rotate_pairs(x, positions, rot):
    """x [tokens, heads, n]: columns 2i and 2i + 1 of the first ``dims`` turn by position * frequency; the others pass."""
    if not rot or not int(rot["dims"]):
        return x
    dims = int(rot["dims"])
    a = positions.to(F64)[:, None, None] * frequencies(rot)
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * torch.cos(a) - v * torch.sin(a)
    out[..., 1:dims:2] = v * torch.cos(a) + u * torch.sin(a)
    return out


def cap(s, softcap):
    return softcap * torch.tanh(s / softcap) if softcap else s


def keys_values(w, p, m, h, positions=None):
    """Rotated keys [T, G, dim] and values [T, G, vdim] of a layer with projections of its own."""
    T, G = h.shape[0], int(m["kv_heads"])
    pos = torch.arange(T) if positions is None else positions
    k = rotate_pairs((h @ w[p + "k"].T).reshape(T, G, int(m["dim"])), pos, m.get("rot"))
    return k, (h @ w[p + "v"].T).reshape(T, G, int(m["vdim"]))


def attention_core(q, k, v, m):
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim] (all rotated) -> heads [T, H * vdim]: causal, capped scores."""
    T, H, G = q.shape[0], int(m["heads"]), int(m["kv_heads"])
    mask = torch.tril(torch.ones(T, T, dtype=torch.bool))
    out = torch.zeros(T, H, v.shape[-1], dtype=F64)
    for hd in range(H):
        g = hd // (H // G)
        s = cap(q[:, hd] @ k[:, g].T * float(m["scale"]), float(m.get("softcap") or 0.0))
        out[:, hd] = torch.softmax(s.masked_fill(~mask, -math.inf), -1) @ v[:, g]
    return out.reshape(T, -1)


def attention(w, p, m, h, kv):
    """``kv``: the (rotated) keys and the values this layer reads, its own or an earlier layer's."""
    T = h.shape[0]
    q = rotate_pairs((h @ w[p + "q"].T).reshape(T, int(m["heads"]), int(m["dim"])), torch.arange(T), m.get("rot"))
    heads = attention_core(q, kv[0], kv[1], m)
    return (heads * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def lightning_core(q, k, v, decay, state=None):
    """q, k [T, H, dim], v [T, H, vdim] (activated): S = decay_h S + k v^T, o = S^T q, one token after the other.  Returns (o, S)."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=F64) if state is None else state.clone()
    d = torch.tensor([float(x) for x in decay], dtype=F64)[:, None, None]
    out = torch.zeros(T, H, v.shape[-1], dtype=F64)
    for t in range(T):
        S = d * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out, S


def lightning(w, p, m, h, eps):
    T, H = h.shape[0], int(m["heads"])
    q, k = (silu(h @ w[p + n].T).reshape(T, H, int(m["dim"])) for n in ("q", "k"))
    v = silu(h @ w[p + "v"].T).reshape(T, H, int(m["vdim"]))
    o, _ = lightning_core(q, k, v, m["decay"])
    o = rms(o.reshape(T, -1), eps) * w[p + "norm"]
    return (o * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def clamped_glu(g, u, limit):
    g, u = g.clamp(max=limit), u.clamp(-limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1.0)


def dense_ff(w, p, mlp, h):
    return clamped_glu(h @ w[p + "gate"].T, h @ w[p + "up"].T, float(mlp["limit"])) @ w[p + "down"].T


def expert(w, p, h):
    return torch.relu(h @ w[p + "up"].T) ** 2 @ w[p + "down"].T


def route(z, correction, router):
    """Router logits of one token -> [(expert, weight)]."""
    E, top, groups = z.shape[0], int(router["top"]), router.get("groups") or dict(count=1, keep=1)
    s = torch.sigmoid(z)
    choice = s + correction
    n, size = int(groups["count"]), E // int(groups["count"])
    rank = sorted(range(n), key=lambda g: (-sum(sorted(choice[g * size:(g + 1) * size].tolist(), reverse=True)[:2]), g))
    allowed = [e for g in rank[:int(groups["keep"])] for e in range(g * size, (g + 1) * size)]
    chosen = sorted(allowed, key=lambda e: (-choice[e].item(), e))[:top]
    total = sum(s[e].item() for e in chosen) + 1e-20
    return [(e, s[e].item() / total * float(router.get("scale", 1.0))) for e in chosen]


def moe(w, p, mlp, h):
    out = torch.zeros_like(h)
    z = h @ w[p + "router"].T
    for t in range(h.shape[0]):
        for e, a in route(z[t], w[p + "correction"], mlp["router"]):
            out[t] += a * expert(w, f"{p}e{e}.", h[t:t + 1])[0]
    return out + expert(w, p + "shared.", h) if mlp.get("shared") else out


def feed_forward(w, p, mlp, h):
    return dense_ff(w, p, mlp, h) if mlp["kind"] == "dense" else moe(w, p, mlp, h)


def layer(w, cfg, i, x, eps, cache):
    """One norm feeds the mixer and the feed-forward; both results are added.  ``cache``: keys and values by layer."""
    p, spec = f"l{i}.", cfg["layers"][i]
    m, h = spec["mixer"], centred_norm(x, w[f"l{i}.norm1"], eps)
    if spec["type"] == "attention":
        src = m.get("kv_from")
        if src is None:
            cache[i] = keys_values(w, p + "mix.", m, h)
        y = attention(w, p + "mix.", m, h, cache[i if src is None else src])
    else:
        y = lightning(w, p + "mix.", m, h, eps)
    if spec.get("mlp"):
        y = y + feed_forward(w, p + "mlp.", spec["mlp"], h)
    return x + y


def forward(weights, cfg, tokens, keep=None):
    """Logits [tokens, vocab] of one whole sequence; ``keep`` receives the stream after every layer."""
    w = {k: v.to(F64) for k, v in weights.items()}
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    cache = {}
    for i in range(len(cfg["layers"])):
        x = layer(w, cfg, i, x, eps, cache)
        if keep is not None:
            keep.append(x.clone())
    return centred_norm(x, w["final.norm"], eps) @ w["embed"].T


# ---- small configurations and random weights for the tests ------------------------------------------------------------
def make_config(vocab=97, width=48, eps=1e-5, layers=("attention/dense", "lightning/moe"), att=None, lin=None, ff=40, limit=1.5, moe=None,
                kv_from=None, per_layer=None):
    """A ``config.json`` dictionary.  ``layers``: per layer "<mixer>/<feed-forward>" with feed-forward dense | moe | none;
    ``kv_from``: {layer: layer whose keys and values it reads}; ``per_layer``: {layer: overrides of the mixer's values}."""
    a = dict(heads=4, kv_heads=2, dim=12, vdim=8, scale=0.3, softcap=5.0, rot=dict(base=1000.0, dims=8, scaling=dict(factor=4.0, low=1.0, high=4.0,
                                                                                                                    original=64)))
    a.update(att or {})
    li = dict(heads=3, dim=8, vdim=12)
    li.update(lin or {})
    mo = dict(ff=16, experts=6, top=2, scale=1.7, groups=dict(count=3, keep=2), shared=20)
    mo.update(moe or {})
    out = []
    for i, kind in enumerate(layers):
        typ, f = kind.split("/")
        mixer = dict(a if typ == "attention" else li, **(per_layer or {}).get(i, {}))
        if typ == "lightning" and "decay" not in mixer:
            n = mixer["heads"]
            mixer["decay"] = [1.0 - 0.5 ** (1 + 9 * (h + i % 2) / (n + 1)) for h in range(n)]
        if kv_from and i in kv_from:
            mixer["kv_from"] = kv_from[i]
        mlp = None
        if f == "dense":
            mlp = dict(kind="dense", ff=ff, limit=limit)
        elif f == "moe":
            mlp = dict(kind="moe", expert=dict(ff=mo["ff"]), router=dict(experts=mo["experts"], top=mo["top"], scale=mo["scale"]))
            if mo["groups"]:
                mlp["router"]["groups"] = mo["groups"]
            if mo["shared"]:
                mlp["shared"] = dict(ff=mo["shared"])
        out.append(dict(type=typ, mixer=mixer, mlp=mlp))
    return dict(architecture="Lapilorn", vocab=vocab, width=width, norm=dict(eps=eps), layers=out)


def random_weights(cfg, seed=0, dtype=torch.bfloat16):
    """Random checkpoint tensors for ``cfg`` (rounded to ``dtype``, so that the oracle and the engine read the same numbers)."""
    gen = torch.Generator().manual_seed(seed)
    W = cfg["width"]
    w = {}

    def lin(name, o, i, s=1.0):
        w[name] = torch.randn(o, i, generator=gen) * s / i ** 0.5
    w["embed"] = torch.randn(cfg["vocab"], W, generator=gen)
    for i, spec in enumerate(cfg["layers"]):
        m, mlp, q, f = spec["mixer"], spec.get("mlp"), f"l{i}.mix.", f"l{i}.mlp."
        w[f"l{i}.norm1"] = torch.randn(W, generator=gen) * 0.2
        nv = m["heads"] * m["vdim"]
        lin(q + "q", m["heads"] * m["dim"], W, 1.5)
        if spec["type"] == "lightning":
            lin(q + "k", m["heads"] * m["dim"], W), lin(q + "v", nv, W)
            w[q + "norm"] = torch.rand(nv, generator=gen) + 0.5
        elif m.get("kv_from") is None:
            lin(q + "k", m["kv_heads"] * m["dim"], W, 1.5), lin(q + "v", m["kv_heads"] * m["vdim"], W)
        lin(q + "g", nv, W), lin(q + "o", W, nv)
        if mlp is None:
            continue
        if mlp["kind"] == "dense":
            lin(f + "gate", mlp["ff"], W, 1.5), lin(f + "up", mlp["ff"], W, 1.5), lin(f + "down", W, mlp["ff"])
            continue
        E, ff = mlp["router"]["experts"], mlp["expert"]["ff"]
        for e in range(E):
            lin(f"{f}e{e}.up", ff, W), lin(f"{f}e{e}.down", W, ff)
        lin(f + "router", E, W)
        w[f + "correction"] = torch.randn(E, generator=gen) * 0.3 - 0.4           # choice scores of both signs
        if mlp.get("shared"):
            lin(f + "shared.up", mlp["shared"]["ff"], W), lin(f + "shared.down", W, mlp["shared"]["ff"])
    w["final.norm"] = torch.randn(W, generator=gen) * 0.2
    return {k: v.to(dtype) for k, v in w.items()}
