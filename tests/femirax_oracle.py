"""A plain, slow Femirax: one function per mechanism, one token or one head at a time, whole sequences, no cache.

Everything runs in the dtype of the weights handed in (the tests use float64 or float32).  Nothing here is shared
with the package: the equations are written out again, in loops where a loop says it most directly.
Shapes: a sequence is x [T, width]; heads are [T, heads, dim].
"""
import math

import torch


# With a generator here every projection's input and output is multiplied by 1 + 2^-9 randn: what rounding activations
# to bfloat16 does to an answer (a head whose output nearly vanishes is divided by its tiny root mean square).
NOISE = None


def linear(x, w):
    if NOISE is None:
        return x @ w.T
    jitter = lambda t: t * (1 + 2.0 ** -9 * torch.randn(t.shape, generator=NOISE, dtype=t.dtype))
    return jitter(jitter(x) @ w.T)


# ------------------------------------------------------------------------------------------- mechanisms
def unit_rms(x, eps):
    """x over its root mean square along the last dimension, eps inside the root."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


def silu(z):
    return z / (1.0 + torch.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rotate(x, base, dims, layout, first_position=0):
    """Rotary positions on the first `dims` of every head of x [T, heads, dim]; row t sits at position
    first_position + t.  layout 'half': i with i + dims/2; 'pairs': 2i with 2i + 1."""
    y = x.clone()
    position = first_position + torch.arange(x.shape[0], dtype=torch.float64)
    for i in range(dims // 2):
        a = position * base ** (-2.0 * i / dims)
        cos, sin = a.cos().to(x.dtype)[:, None], a.sin().to(x.dtype)[:, None]
        j0, j1 = (i, i + dims // 2) if layout == "half" else (2 * i, 2 * i + 1)
        u, v = x[:, :, j0], x[:, :, j1]
        y[:, :, j0] = u * cos - v * sin
        y[:, :, j1] = v * cos + u * sin
    return y


def causal_attention(q, k, v, scale):
    """q [T, H, d], k and v [T, G, d]: query head h reads key/value head h // (H / G)."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = q.new_zeros(T, H, v.shape[-1])
    hidden = torch.ones(T, T, dtype=torch.bool).triu(1)             # key j > query i
    for h in range(H):
        g = h // (H // G)
        s = ((q[:, h] @ k[:, g].T) * scale).masked_fill(hidden, -math.inf)
        p = torch.exp(s - s.max(-1, keepdim=True).values)
        out[:, h] = (p / p.sum(-1, keepdim=True)) @ v[:, g]
    return out


def decayed_state(q, k, v, alpha):
    """The linear recurrence, token by token: S <- diag(alpha_t) S + k_t v_t^T, o_t = S^T q_t, from S = 0.
    q, k, alpha [T, H, dk]; v [T, H, dv]."""
    T, H, dk = q.shape
    S = q.new_zeros(H, dk, v.shape[-1])
    out = q.new_zeros(T, H, v.shape[-1])
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out


def retention(h, w, cfg, eps):
    T, H, dk, dv = h.shape[0], cfg["heads"], cfg["dim"], cfg["vdim"]
    rot = cfg["rot"]
    q = rotate(linear(h, w["q"]).view(T, H, dk), rot["base"], rot["dims"], "half")
    k = rotate(linear(h, w["k"]).view(T, H, dk), rot["base"], rot["dims"], "half") * dk ** -0.5
    v = linear(h, w["v"]).view(T, H, dv)
    alpha = torch.tensor(cfg["decay"], dtype=h.dtype).view(1, H, 1).expand(T, H, dk)
    o = unit_rms(decayed_state(q, k, v, alpha), eps).reshape(T, H * dv)
    return linear(o * silu(linear(h, w["g"])), w["o"])


def key_value_attention(h, w, cfg, eps):
    T, H, G, d = h.shape[0], cfg["heads"], cfg["kv_heads"], cfg["dim"]
    rot = cfg["rot"]
    raw = linear(h, w["k"]).view(T, G, d)
    q = unit_rms(rotate(linear(h, w["q"]).view(T, H, d), rot["base"], rot["dims"], "pairs"), eps)
    k = unit_rms(rotate(raw, rot["base"], rot["dims"], "pairs"), eps)
    return linear(causal_attention(q, k, raw, cfg["scale"]).reshape(T, H * d), w["o"])


def channel_decay(h, a1, a2, b, tau):
    z = linear(h, a1) @ a2.T + b
    return (1.0 / (1.0 + torch.exp(-z))) ** (1.0 / tau)


def gated_linear(h, w, cfg, eps):
    T, H, dk, dv = h.shape[0], cfg["heads"], cfg["dim"], cfg["vdim"]
    q = linear(h, w["q"]).view(T, H, dk) * dk ** -0.5
    k = linear(h, w["k"]).view(T, H, dk)
    v = linear(h, w["v"]).view(T, H, dv)
    alpha = channel_decay(h, w["a1"], w["a2"], w["a2.b"], cfg["tau"]).view(T, H, dk)
    o = rms_norm(decayed_state(q, k, v, alpha), w["norm"], eps).reshape(T, H * dv)
    return linear(o * silu(linear(h, w["g"])), w["o"])


def _sub(w, prefix):
    return {n[len(prefix):]: t for n, t in w.items() if n.startswith(prefix)}


def parallel(h, w, cfg, eps):
    left = key_value_attention(h, _sub(w, "left."), cfg["left"], eps)
    right = gated_linear(h, _sub(w, "right."), cfg["right"], eps)
    return 0.5 * (rms_norm(left, w["left.out"], eps) + rms_norm(right, w["right.out"], eps))


def dense_mlp(h, w):
    return linear(silu(linear(h, w["gate"])) * linear(h, w["up"]), w["down"])


def token_side(x, tokens, table, layer, dim, w, eps):
    e = table[tokens][:, layer * dim:(layer + 1) * dim]
    y = linear(gelu_tanh(linear(x, w["gate"])) * e, w["proj"])
    return rms_norm(y, w["norm"], eps)


# ------------------------------------------------------------------------------------------- the model
def forward(tokens, config, weights, layers_out=None):
    """Logits [T, vocab] of one whole sequence.  `layers_out`: a list that receives the residual after each layer."""
    eps, sdim = config["norm"]["eps"], config["token_side"]["dim"]
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    x = weights["embed"][tokens]
    for i, layer in enumerate(config["layers"]):
        w = _sub(weights, f"l{i}.")
        mix = retention if layer["type"] == "retention" else parallel
        x = x + mix(rms_norm(x, w["norm1"], eps), _sub(w, "mix."), layer["mixer"], eps)
        if layer["mlp"] is not None:
            x = x + dense_mlp(rms_norm(x, w["norm2"], eps), _sub(w, "mlp."))
        x = x + token_side(x, tokens, weights["side.embed"], i, sdim, _sub(w, "side."), eps)
        if layers_out is not None:
            layers_out.append(x)
    return linear(rms_norm(x, weights["final.norm"], eps), weights["head"])


def greedy(prompt, n, config, weights):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(toks, config, weights)[-1].argmax()))
    return toks[len(prompt):]


# ------------------------------------------------------------------------------------------- test models
def tensor_shapes(config, rank):
    """Name -> shape of every tensor of a model; `rank`: inner size of the low-rank decay projections."""
    W, V, sd = config["width"], config["vocab"], config["token_side"]["dim"]
    out = {"embed": (V, W), "side.embed": (V, sd * len(config["layers"])), "final.norm": (W,), "head": (V, W)}
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        out[p + "norm1"] = (W,)
        if layer["type"] == "retention":
            H, dk, dv = m["heads"], m["dim"], m["vdim"]
            out.update({p + "mix.q": (H * dk, W), p + "mix.k": (H * dk, W), p + "mix.v": (H * dv, W),
                        p + "mix.g": (H * dv, W), p + "mix.o": (W, H * dv)})
        else:
            L, R = m["left"], m["right"]
            H, dk, dv = R["heads"], R["dim"], R["vdim"]
            q = p + "mix.right."
            out.update({p + "mix.left.q": (L["heads"] * L["dim"], W), p + "mix.left.k": (L["kv_heads"] * L["dim"], W),
                        p + "mix.left.o": (W, L["heads"] * L["dim"]), q + "q": (H * dk, W), q + "k": (H * dk, W),
                        q + "v": (H * dv, W), q + "g": (H * dv, W), q + "o": (W, H * dv), q + "norm": (dv,),
                        q + "a1": (rank, W), q + "a2": (H * dk, rank), q + "a2.b": (H * dk,),
                        p + "mix.left.out": (W,), q + "out": (W,)})
        if layer["mlp"] is not None:
            ff = layer["mlp"]["ff"]
            out.update({p + "norm2": (W,), p + "mlp.gate": (ff, W), p + "mlp.up": (ff, W), p + "mlp.down": (W, ff)})
        out.update({p + "side.gate": (sd, W), p + "side.proj": (W, sd), p + "side.norm": (W,)})
    return out


def random_weights(config, rank=6, seed=0, decay_bias=3.0):
    """bfloat16 weights of a sensible scale: linear maps keep the variance, norm weights sit around one, the decay
    projection's bias around `decay_bias`."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(config, rank).items():
        r = torch.randn(shape, generator=g)
        if name.endswith(".a2.b"):
            t = decay_bias + r
        elif len(shape) == 1:
            t = 1.0 + 0.2 * r
        elif name in ("embed", "side.embed"):
            t = r
        else:
            t = r * shape[1] ** -0.5
        out[name] = t.to(torch.bfloat16)
    return out
