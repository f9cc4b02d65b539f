"""The Mamevik decoder stated plainly: whole sequences, no cache, no batching, one function per mechanism.

Written from the design's equations in this file's own notation; it shares no code with the product.
``forward(config, weights, tokens)`` returns the logits at every position (in the dtype of the weights:
tests use float64).  ``config`` is the dict a model folder's config.json holds.  Notation: T tokens, E stream
width, H heads, D query/key size, V value size, R latent size, W window, G groups of B and C, N state size,
I = H V inner width of the recurrence, F inner width of an expert, X experts.

    x_0 = N_embed(table[token] + pairs[row(previous token, token)])
    layers in order; those of the loop as often as it says, each pass begun with  x <- W_in [x; x_0] + step[pass]
    per layer   x <- x + mixer(N_1(x));  x <- x + experts(N_2(x))        (layers with a feed-forward)
    logits = cap * tanh(scale * table @ N_final(x) / cap)
    N(x) = x / sqrt(mean(x^2) + eps) * (1 + w)
"""
from __future__ import annotations

import math

import torch


# ---- configurations and weights of the tests --------------------------------------------------------
def mamba_layer(*, heads, vdim, state, groups=1, conv=4, norm_groups=1, mlp=None):
    return dict(type="mamba2", mixer=dict(heads=heads, vdim=vdim, state=state, groups=groups, conv=conv,
                                          norm_groups=norm_groups), mlp=mlp)


def attention_layer(*, heads, dim, vdim, kv_rank, window, scale=None, mlp=None):
    mixer = dict(heads=heads, dim=dim, vdim=vdim, kv_rank=kv_rank, scale=dim ** -0.5 if scale is None else scale,
                 mask=dict(size=window))
    return dict(type="latent_attention", mixer=mixer, mlp=mlp)


def moe(*, experts, top, ff, limit):
    return dict(kind="moe", expert=dict(ff=ff, limit=limit), router=dict(experts=experts, top=top))


def model_config(layers, *, vocab, width, loop, bigram, eps=1e-5, logit_scale=1.0, softcap=20.0):
    """``loop`` (start, stop, times); ``bigram`` (buckets, factor of the previous token, factor of the token)."""
    return dict(architecture="Mamevik", vocab=vocab, width=width, norm=dict(eps=eps), layers=[dict(l) for l in layers],
                loop=dict(start=loop[0], stop=loop[1], times=loop[2]),
                embedding=dict(bigram=dict(buckets=bigram[0], mul_prev=bigram[1], mul_cur=bigram[2])),
                logit_scale=logit_scale, logit_softcap=softcap)


def tensor_shapes(cfg):
    E = cfg["width"]
    shapes = {"embed": (cfg["vocab"], E), "bigram": (cfg["embedding"]["bigram"]["buckets"] + 1, E),
              "embed.norm": (E,), "final.norm": (E,), "loop.in": (E, 2 * E), "loop.step": (cfg["loop"]["times"], E)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        shapes[p + "norm1"] = (E,)
        H, V = m["heads"], m["vdim"]
        if layer["type"] == "mamba2":
            channels = H * V + 2 * m["groups"] * m["state"]
            shapes.update({p + "mix.in": (H * V + channels + H, E), p + "mix.conv": (channels, m["conv"]),
                           p + "mix.conv.b": (channels,), p + "mix.dt_bias": (H,), p + "mix.A_log": (H,),
                           p + "mix.D": (H,), p + "mix.norm": (H * V,), p + "mix.o": (E, H * V)})
        else:
            D, R = m["dim"], m["kv_rank"]
            shapes.update({p + "mix.q": (H * D, E), p + "mix.dkv": (R, E), p + "mix.dkv.norm": (R,),
                           p + "mix.uk": (H * D, R), p + "mix.uv": (H * V, R), p + "mix.sink": (H,),
                           p + "mix.o": (E, H * V)})
        mlp = layer.get("mlp")
        if mlp is not None:
            shapes[p + "norm2"] = (E,)
            F, X = mlp["expert"]["ff"], mlp["router"]["experts"]
            for e in range(X):
                shapes.update({f"{p}mlp.e{e}.gate": (F, E), f"{p}mlp.e{e}.up": (F, E), f"{p}mlp.e{e}.down": (E, F)})
            shapes.update({p + "mlp.router": (X, E), p + "mlp.router.b": (X,)})
    return shapes


def random_weights(cfg, seed, dtype=torch.float32):
    """Weights that keep every mechanism alive: norm weights around zero (or around one where the weight is
    plain), decays that reach from a few tokens to hundreds, routers that spread their choices."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.rsplit(".", 1)[-1]
        if leaf in ("norm1", "norm2") or name in ("final.norm", "embed.norm"):
            t = 0.2 * torch.randn(shape, generator=g)
        elif name.endswith("mix.norm") or name.endswith("dkv.norm"):
            t = 1.0 + 0.2 * torch.randn(shape, generator=g)
        elif leaf == "A_log":
            t = torch.empty(shape).uniform_(-3.0, 1.0, generator=g)
        elif leaf == "dt_bias":
            t = torch.empty(shape).uniform_(-3.0, 0.5, generator=g)
        elif leaf == "D":
            t = 0.5 + 0.5 * torch.randn(shape, generator=g)
        elif leaf == "sink":
            t = torch.randn(shape, generator=g)
        elif name.endswith("router.b") or name.endswith("conv.b"):
            t = 0.3 * torch.randn(shape, generator=g)
        elif leaf == "conv":
            t = torch.randn(shape, generator=g) / math.sqrt(shape[-1])
        elif leaf == "router":      # decisive routers: few close calls between experts that weigh much
            t = 4.0 * torch.randn(shape, generator=g) / math.sqrt(shape[-1])
        elif name in ("embed", "bigram"):
            t = torch.randn(shape, generator=g)
        elif name == "loop.step":
            t = 0.5 * torch.randn(shape, generator=g)
        else:
            t = torch.randn(shape, generator=g) / math.sqrt(shape[-1])
        # what a bfloat16 file would hold, so that a 64-bit evaluation and a loaded model see one model
        out[name] = t.to(torch.bfloat16).to(dtype)
    return out


# ---- mechanisms ---------------------------------------------------------------------------------------
def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def zero_centred_norm(x, w, eps):
    return unit_rms(x, eps) * (1.0 + w)


def silu(z):
    return z * torch.sigmoid(z)


def pair_rows(tokens, b):
    """The row of the pair table of every token: its own where nothing is in front, else the pair's bucket."""
    rows = []
    for i, token in enumerate(tokens.tolist()):
        rows.append(b["buckets"] if i == 0
                    else (int(tokens[i - 1]) * b["mul_prev"] + token * b["mul_cur"]) % b["buckets"])
    return torch.tensor(rows, dtype=torch.long)


def embed(tokens, cfg, w, *, leave_out=()):
    x = w["embed"][tokens]
    if "bigram" not in leave_out:
        x = x + w["bigram"][pair_rows(tokens, cfg["embedding"]["bigram"])]
    return zero_centred_norm(x, w["embed.norm"], cfg["norm"]["eps"])


def causal_conv(u, taps, bias):
    """y_t[c] = bias[c] + sum_j taps[c, j] u_{t - (K - 1) + j}[c], nothing in front of the first token."""
    T, K = u.shape[0], taps.shape[1]
    padded = torch.cat([torch.zeros(K - 1, u.shape[1], dtype=u.dtype), u])
    return bias + sum(padded[j:j + T] * taps[:, j] for j in range(K))


def state_space(x, B, C, dt, a, D):
    """Per head S_t = a_t S_{t-1} + dt_t B_t x_t^T, y_t = S_t^T C_t + D x_t; x [T, H, V], B and C [T, G, N],
    dt and a [T, H], D [H]; head h reads group h // (H / G)."""
    T, H, V = x.shape
    G, N = B.shape[1:]
    S = torch.zeros(H, N, V, dtype=x.dtype)
    Bh, Ch = B.repeat_interleave(H // G, 1), C.repeat_interleave(H // G, 1)
    out = torch.zeros_like(x)
    for t in range(T):
        S = a[t][:, None, None] * S + dt[t][:, None, None] * Bh[t][:, :, None] * x[t][:, None, :]
        out[t] = (S * Ch[t][:, :, None]).sum(1) + D[:, None] * x[t]
    return out


def gated_group_norm(y, z, w, groups, eps):
    """The gate first, then the norm of equal parts, each by its own root mean square."""
    T, width = y.shape
    y = y * silu(z)
    return unit_rms(y.view(T, groups, width // groups), eps).reshape(T, width) * w


def mamba2(h, m, w, p, eps, leave_out=()):
    T = h.shape[0]
    H, V, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * V
    z, u, dt = torch.split(h @ w[p + "in"].T, [inner, inner + 2 * G * N, H], -1)
    taps = w[p + "conv"]
    if "conv" in leave_out:
        taps = torch.cat([torch.zeros_like(taps[:, :-1]), taps[:, -1:]], 1)
    u = silu(causal_conv(u, taps, w[p + "conv.b"]))
    x, B, C = torch.split(u, [inner, G * N, G * N], -1)
    dt = torch.nn.functional.softplus(dt + w[p + "dt_bias"], threshold=1e6)
    a = torch.exp(-torch.exp(w[p + "A_log"]) * dt)
    D = torch.zeros_like(w[p + "D"]) if "D" in leave_out else w[p + "D"]
    y = state_space(x.reshape(T, H, V), B.reshape(T, G, N), C.reshape(T, G, N), dt, a, D).reshape(T, inner)
    return gated_group_norm(y, z, w[p + "norm"], m["norm_groups"], eps) @ w[p + "o"].T


def latent_attention(h, m, w, p, eps, leave_out=()):
    T = h.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).view(T, H, D)
    c = unit_rms(h @ w[p + "dkv"].T, eps) * w[p + "dkv.norm"]
    k = (c @ w[p + "uk"].T).view(T, H, D)
    v = (c @ w[p + "uv"].T).view(T, H, V)
    distance = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    seen = distance >= 0
    if m.get("mask") and "mask" not in leave_out:
        seen = seen & (distance < m["mask"]["size"])
    score = torch.einsum("ihd,jhd->hij", q, k) * m["scale"]
    score = score.masked_fill(~seen, -math.inf)
    sink = w[p + "sink"][:, None, None]
    if "sink" in leave_out:
        weights = torch.softmax(score, -1)
    else:
        top = torch.maximum(score.amax(-1, keepdim=True), sink)
        e = torch.exp(score - top)
        weights = e / (e.sum(-1, keepdim=True) + torch.exp(sink - top))
    return torch.einsum("hij,jhv->ihv", weights, v).reshape(T, H * V) @ w[p + "o"].T


STAKE_FLOOR = 0.02      # a close call between experts that both weigh less than this is no close call


def route(h, mlp, w, p, leave_out=()):
    """Chosen experts [T, top] and their weights; also the margin of every token's choice: the gap between the
    last chosen and the first refused logit (infinite where what is at stake weighs next to nothing)."""
    top = mlp["router"]["top"]
    z = h @ w[p + "router"].T
    if "router.b" not in leave_out:
        z = z + w[p + "router.b"]
    order = torch.sort(z, -1, descending=True)
    ids, weights = order.indices[:, :top], torch.softmax(order.values[:, :top], -1)
    margin = torch.full((h.shape[0],), math.inf, dtype=h.dtype)
    if top < z.shape[1]:
        gap = order.values[:, top - 1] - order.values[:, top]
        margin = torch.where(weights[:, -1] > STAKE_FLOOR, gap, margin)
    return ids, weights, margin


def clamped_unit(h, gate, up, down, limit):
    g = torch.clamp(h @ gate.T, max=limit)
    u = torch.clamp(h @ up.T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ down.T


def experts(h, mlp, w, p, leave_out=()):
    ids, weights, margin = route(h, mlp, w, p, leave_out)
    limit = 1e9 if "limit" in leave_out else mlp["expert"]["limit"]
    out = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        token, slot = (ids == e).nonzero(as_tuple=True)
        if len(token):
            q = f"{p}e{e}."
            out[token] += weights[token, slot, None] * clamped_unit(h[token], w[q + "gate"], w[q + "up"], w[q + "down"], limit)
    return out, margin


def layer_order(cfg):
    """(layer, pass number if the layer begins a pass of the loop else None) in running order."""
    loop, count = cfg["loop"], len(cfg["layers"])
    order = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        order += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return order + [(i, None) for i in range(loop["stop"], count)]


def forward(cfg, w, tokens, *, streams=None, margins=None, leave_out=()):
    """Logits [T, vocab].  ``streams`` (a list) receives the stream after every layer run; ``margins`` (a list)
    the routers' smallest margin at every position; ``leave_out`` names mechanisms to drop (tests use it to show
    that each one moves the logits)."""
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    eps = cfg["norm"]["eps"]
    x0 = x = embed(tokens, cfg, w, leave_out=leave_out)
    worst = torch.full((len(tokens),), math.inf, dtype=x.dtype)
    for i, begins in layer_order(cfg):
        p, layer = f"l{i}.", cfg["layers"][i]
        if begins is not None:
            if "loop.in" not in leave_out:
                x = torch.cat([x, x0], -1) @ w["loop.in"].T
            if "loop.step" not in leave_out:
                x = x + w["loop.step"][begins]
        mixer = mamba2 if layer["type"] == "mamba2" else latent_attention
        x = x + mixer(zero_centred_norm(x, w[p + "norm1"], eps), layer["mixer"], w, p + "mix.", eps, leave_out)
        if layer.get("mlp") is not None:
            f, margin = experts(zero_centred_norm(x, w[p + "norm2"], eps), layer["mlp"], w, p + "mlp.", leave_out)
            worst = torch.minimum(worst, margin)
            x = x + f
        if streams is not None:
            streams.append(x.clone())
    if margins is not None:
        margins.append(worst)
    logits = zero_centred_norm(x, w["final.norm"], eps) @ w["embed"].T * cfg["logit_scale"]
    if "softcap" in leave_out:
        return logits
    return cfg["logit_softcap"] * torch.tanh(logits / cfg["logit_softcap"])
