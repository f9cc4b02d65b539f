"""The Tabopel decoder stated plainly: whole sequences, no cache, no batching, one function per mechanism.

Written from the design's equations in this file's own notation; it shares no code with the product.
``forward(config, weights, tokens)`` returns the logits at every position (in the dtype of the weights:
tests use float64).  ``config`` is the dict a model folder's config.json holds.  Notation: T tokens, E stream
width, H query heads, G key/value heads, D query/key size, V value size, F inner width of a feed-forward,
X experts with tensors, I experts that hand their input on, K taps.

    x = c * table[token]
    layers in order; those of the loop as often as it says, each pass begun with  x <- x + step[pass]
    per layer   x <- x + N_1b(mixer(N_1(x)));  x <- x + N_2b(ff(N_2(x)))        (layers with a feed-forward)
    logits = head @ N_final(x)
    N(x) = x / sqrt(mean(x^2) + eps) * w
"""
from __future__ import annotations

import math

import torch


# ---- configurations and weights of the tests --------------------------------------------------------
def rotation(dims, base, scaling=None):
    rot = dict(base=base, dims=dims)
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return rot


def conv_attention(*, heads, kv_heads, dim, vdim, conv, rot, scale=None, mlp=None):
    return dict(type="attention", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv, rot=rot,
                                             scale=dim ** -0.5 if scale is None else scale), mlp=mlp)


def capped_attention(*, heads, kv_heads, dim, vdim, rot, softcap, scale=None, mlp=None):
    return dict(type="attention_2", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, rot=rot, softcap=softcap,
                                               scale=dim ** -0.5 if scale is None else scale), mlp=mlp)


def retention(*, dim, vdim, decay, rot, mlp=None):
    return dict(type="retention", mixer=dict(heads=len(decay), dim=dim, vdim=vdim, decay=list(decay), rot=rot), mlp=mlp)


def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(*, experts, top, ff, identity):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top, identity=identity))


def model_config(layers, *, vocab, width, loop=None, eps=1e-5, scale=1.0):
    """``loop`` (start, stop, times), or None."""
    cfg = dict(architecture="Tabopel", vocab=vocab, width=width, norm=dict(eps=eps), embedding=dict(scale=scale),
               layers=[dict(l) for l in layers])
    if loop is not None:
        cfg["loop"] = dict(start=loop[0], stop=loop[1], times=loop[2])
    return cfg


def tensor_shapes(cfg):
    E = cfg["width"]
    shapes = {"embed": (cfg["vocab"], E), "head": (cfg["vocab"], E), "final.norm": (E,)}
    if cfg.get("loop"):
        shapes["loop.step"] = (cfg["loop"]["times"], E)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        H, D, V = m["heads"], m["dim"], m["vdim"]
        G = m.get("kv_heads", H)
        shapes.update({p + "norm1": (E,), p + "norm1b": (E,), p + "mix.q": (H * D, E), p + "mix.k": (G * D, E),
                       p + "mix.v": (G * V, E), p + "mix.o": (E, H * V)})
        if layer["type"] == "attention":
            K = m["conv"]
            shapes.update({p + "mix.q.conv": (H * D, K), p + "mix.k.conv": (G * D, K), p + "mix.v.conv": (G * V, K),
                           p + "mix.g": (H * V, E)})
        elif layer["type"] == "attention_2":
            shapes.update({p + "mix.q.b": (H * D,), p + "mix.k.b": (G * D,), p + "mix.v.b": (G * V,),
                           p + "mix.q.norm": (H * D,), p + "mix.k.norm": (G * D,), p + "mix.sink": (H,)})
        else:
            shapes[p + "mix.g"] = (H * V, E)
        mlp = layer.get("mlp")
        if mlp is None:
            continue
        shapes.update({p + "norm2": (E,), p + "norm2b": (E,)})
        if mlp["kind"] == "dense":
            shapes.update({p + "mlp.up": (mlp["ff"], E), p + "mlp.down": (E, mlp["ff"])})
            continue
        F, X, I = mlp["expert"]["ff"], mlp["router"]["experts"], mlp["router"]["identity"]
        for e in range(X):
            shapes.update({f"{p}mlp.e{e}.up": (F, E), f"{p}mlp.e{e}.down": (E, F)})
        shapes.update({p + "mlp.router": (X + I, E), p + "mlp.correction": (X + I,)})
    return shapes


def random_weights(cfg, seed, dtype=torch.float32):
    """Weights that keep every mechanism alive: scores that reach into the cap, sinks that weigh, routers that
    spread their choices, corrections that change them."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.rsplit(".", 1)[-1]
        if "norm" in leaf:
            t = 1.0 + 0.3 * torch.randn(shape, generator=g)
        elif leaf == "sink":
            t = 1.0 + torch.randn(shape, generator=g)
        elif leaf == "b":
            t = 0.4 * torch.randn(shape, generator=g)
        elif leaf == "conv":
            t = torch.randn(shape, generator=g) / math.sqrt(shape[-1])
        elif leaf == "router":      # decisive routers: few close calls between experts that weigh much
            t = 3.0 * torch.randn(shape, generator=g) / math.sqrt(shape[-1])
        elif leaf == "correction":
            t = 0.1 * torch.randn(shape, generator=g)
        elif name == "embed":
            t = torch.randn(shape, generator=g)
        elif name == "loop.step":
            t = 0.5 * torch.randn(shape, generator=g)
        elif leaf in ("q", "k"):
            t = 1.5 * torch.randn(shape, generator=g) / math.sqrt(shape[-1])
        else:
            t = torch.randn(shape, generator=g) / math.sqrt(shape[-1])
        # what a bfloat16 file would hold, so that a 64-bit evaluation and a loaded model see one model
        out[name] = t.to(torch.bfloat16).to(dtype)
    return out


# ---- mechanisms ---------------------------------------------------------------------------------------
def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    return unit_rms(x, eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def causal_conv(u, taps):
    """y_t[c] = sum_j taps[c, j] u_{t - (K - 1) + j}[c], nothing in front of the first token."""
    T, K = u.shape[0], taps.shape[1]
    padded = torch.cat([torch.zeros(K - 1, u.shape[1], dtype=u.dtype), u])
    return sum(padded[j:j + T] * taps[:, j] for j in range(K))


def frequencies(rot):
    """One frequency a pair, base^(-2i/dims); with scaling, by the wavelength against the original length."""
    n = rot["dims"]
    scaling, out = rot.get("scaling"), []
    for i in range(n // 2):
        f = rot["base"] ** (-2.0 * i / n)
        if scaling:
            turns = scaling["original"] * f / (2.0 * math.pi)        # original length over wavelength
            if turns < scaling["low"]:
                f = f / scaling["factor"]
            elif turns <= scaling["high"]:
                s = (turns - scaling["low"]) / (scaling["high"] - scaling["low"])
                f = (1.0 - s) * f / scaling["factor"] + s * f
        out.append(f)
    return torch.tensor(out, dtype=torch.float64)


def rotate(x, rot, positions=None):
    """x [T, heads, D]: entry i of the first ``dims`` and entry i + dims/2 form a pair, turned by position * f_i."""
    n = rot["dims"] if rot else 0
    if not n:
        return x
    positions = torch.arange(x.shape[0]) if positions is None else positions
    angle = (positions.double()[:, None] * frequencies(rot)).to(x.dtype)[:, None, :]
    c, s = torch.cos(angle), torch.sin(angle)
    u, v = x[..., :n // 2], x[..., n // 2:n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., n:]], -1)


def softcap(score, cap):
    return cap * torch.tanh(score / cap)


def weigh(score, sink):
    """exp(score) / (exp(sink) + sum exp(score)) over the last axis of score [H, T, T] (-inf: not seen)."""
    sink = sink[:, None, None]
    top = torch.maximum(score.amax(-1, keepdim=True), sink)
    e = torch.exp(score - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - top))


def attend(q, k, v, scale, *, cap=None, sink=None):
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H V]; query head h reads key/value head h // (H / G)."""
    T, H = q.shape[:2]
    share = H // k.shape[1]
    k, v = k.repeat_interleave(share, 1), v.repeat_interleave(share, 1)
    score = torch.einsum("ihd,jhd->hij", q, k) * scale
    if cap is not None:
        score = softcap(score, cap)
    ahead = torch.arange(T)[None, :] > torch.arange(T)[:, None]
    score = score.masked_fill(ahead, -math.inf)
    weights = torch.softmax(score, -1) if sink is None else weigh(score, sink)
    return torch.einsum("hij,jhv->ihv", weights, v).reshape(T, -1)


def attention(h, m, w, p, eps, leave_out=()):
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (h @ w[p + n].T for n in "qkv")
    if "conv" not in leave_out:
        q, k, v = (causal_conv(u, w[f"{p}{n}.conv"]) for n, u in zip("qkv", (q, k, v)))
    rot = dict(m["rot"])
    if "scaling" in leave_out:
        rot.pop("scaling", None)
    q, k = rotate(q.view(T, H, D), rot), rotate(k.view(T, G, D), rot)
    one = None if "sink" in leave_out else torch.zeros(H, dtype=h.dtype)      # exp(0) in the denominator
    o = attend(q, k, v.view(T, G, V), m["scale"], sink=one)
    if "g" not in leave_out:
        o = o * torch.sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


def attention_2(h, m, w, p, eps, leave_out=()):
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (h @ w[p + n].T + (0.0 if "b" in leave_out else w[f"{p}{n}.b"]) for n in "qkv")
    if "qk_norm" not in leave_out:
        q, k = norm(q, w[p + "q.norm"], eps), norm(k, w[p + "k.norm"], eps)
    q, k = rotate(q.view(T, H, D), m["rot"]), rotate(k.view(T, G, D), m["rot"])
    o = attend(q, k, v.view(T, G, V), m["scale"], cap=None if "softcap" in leave_out else m["softcap"],
               sink=None if "sink" in leave_out else w[p + "sink"])
    return o @ w[p + "o"].T


def decayed_memory(q, k, v, decay):
    """Per head S_t = decay S_{t-1} + k_t v_t^T, o_t = S_t^T q_t; q and k [T, H, D], v [T, H, V], decay [H]."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=q.dtype)
    out = torch.zeros_like(v)
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out


def retain(h, m, w, p, eps, leave_out=()):
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k, v = (h @ w[p + n].T for n in "qkv")
    rot = None if "retention.rot" in leave_out else m["rot"]
    q, k = rotate(q.view(T, H, D), rot), rotate(k.view(T, H, D), rot) * D ** -0.5
    o = decayed_memory(q, k, v.view(T, H, V), torch.tensor(m["decay"], dtype=h.dtype))
    o = unit_rms(o, eps).reshape(T, H * V)
    return (o * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def unit(h, up, down):
    """Two products with the squared positive part between them."""
    return torch.relu(h @ up.T) ** 2 @ down.T


STAKE_FLOOR = 0.01      # a close call between experts that both weigh less than this is no close call


def route(h, mlp, w, p, leave_out=()):
    """Chosen experts [T, top] and their weights; also the margin of every token's choice: the gap between the
    last chosen and the first refused choice score, relative to that score's own size (infinite where what is at
    stake weighs next to nothing)."""
    top = mlp["router"]["top"]
    s = torch.softmax(h @ w[p + "router"].T, -1)
    choice = s if "correction" in leave_out else s + w[p + "correction"]
    order = torch.sort(choice, -1, descending=True)
    ids = order.indices[:, :top]
    weights = torch.gather(s, 1, ids)
    margin = torch.full((h.shape[0],), math.inf, dtype=h.dtype)
    if top < s.shape[1]:
        gap = order.values[:, top - 1] - order.values[:, top]
        at_stake = torch.maximum(weights[:, -1], torch.gather(s, 1, order.indices[:, top:top + 1])[:, 0])
        margin = torch.where(at_stake > STAKE_FLOOR, gap / at_stake, margin)
    return ids, weights, margin


def experts(h, mlp, w, p, leave_out=()):
    ids, weights, margin = route(h, mlp, w, p, leave_out)
    X = mlp["router"]["experts"]
    out = torch.zeros_like(h)
    for e in range(X + mlp["router"]["identity"]):
        token, slot = (ids == e).nonzero(as_tuple=True)
        if not len(token):
            continue
        if e >= X:
            y = torch.zeros_like(h[token]) if "identity" in leave_out else h[token]
        else:
            y = unit(h[token], w[f"{p}e{e}.up"], w[f"{p}e{e}.down"])
        out[token] += weights[token, slot, None] * y
    return out, margin


def layer_order(cfg):
    """(layer, pass number if the layer begins a pass of the loop else None) in running order."""
    loop, count = cfg.get("loop"), len(cfg["layers"])
    if not loop:
        return [(i, None) for i in range(count)]
    order = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        order += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return order + [(i, None) for i in range(loop["stop"], count)]


MIXERS = dict(attention=attention, attention_2=attention_2, retention=retain)


def forward(cfg, w, tokens, *, streams=None, margins=None, leave_out=()):
    """Logits [T, vocab].  ``streams`` (a list) receives the stream after every layer run; ``margins`` (a list)
    the routers' smallest margin at every position; ``leave_out`` names mechanisms to drop (tests use it to show
    that each one moves the logits)."""
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    eps = cfg["norm"]["eps"]
    x = w["embed"][tokens] * cfg["embedding"]["scale"]
    worst = torch.full((len(tokens),), math.inf, dtype=x.dtype)
    for i, begins in layer_order(cfg):
        p, layer = f"l{i}.", cfg["layers"][i]
        if begins is not None and "loop.step" not in leave_out:
            x = x + w["loop.step"][begins]
        y = MIXERS[layer["type"]](norm(x, w[p + "norm1"], eps), layer["mixer"], w, p + "mix.", eps, leave_out)
        x = x + norm(y, w[p + "norm1b"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            h = norm(x, w[p + "norm2"], eps)
            if mlp["kind"] == "dense":
                f = unit(h, w[p + "mlp.up"], w[p + "mlp.down"])
            else:
                f, margin = experts(h, mlp, w, p + "mlp.", leave_out)
                worst = torch.minimum(worst, margin)
            x = x + norm(f, w[p + "norm2b"], eps)
        if streams is not None:
            streams.append(x.clone())
    if margins is not None:
        margins.append(worst)
    return norm(x, w["final.norm"], eps) @ w["head"].T
