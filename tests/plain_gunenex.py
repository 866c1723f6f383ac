"""A plain, slow implementation of the Gunenex decoder from its equations: one function per mechanism, whole sequences at
a time, double precision, loops where a loop is the clearest way to say it.  It shares nothing with the engine (no part,
no kernel, no cache): the tests compare the engine with it.

A model is (config dict, {tensor name: torch tensor}).  Tensor names: `embed`, `final.norm`, `head`, and per layer i
`l<i>.norm1`, `l<i>.norm2`, `l<i>.mix.*`, `l<i>.mlp.*`, `l<i>.hc1.*`, `l<i>.hc2.*`.
"""
import torch

F = torch.float64


# ----------------------------------------------------------------------------- small pieces
def rms_norm(x, w, eps):
    """x over its root mean square along the last axis, times w (a vector, a single number, or None)."""
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.where(z > 30, z, torch.log1p(torch.exp(torch.clamp(z, max=30))))


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def rotate_halves(x, dims, base):
    """x [T, heads, n]: of each head's first `dims` entries, i and i + dims/2 turn together by position * base^(-2i/dims)."""
    out = x.clone()
    pos = torch.arange(x.shape[0], dtype=F)
    for i in range(dims // 2):
        ang = pos * base ** (-2.0 * i / dims)
        c, s = torch.cos(ang)[:, None], torch.sin(ang)[:, None]
        a, b = i, i + dims // 2
        out[..., a] = x[..., a] * c - x[..., b] * s
        out[..., b] = x[..., b] * c + x[..., a] * s
    return out


def causal_conv(x, taps):
    """x [T, C], taps [C, n]: y[t] = sum_j taps[:, j] * x[t - n + 1 + j], zeros before the start."""
    T, n = x.shape[0], taps.shape[1]
    y = torch.zeros_like(x)
    for j in range(n):
        back = n - 1 - j                                                # how many tokens before the current one
        if back < T:
            y[back:] += taps[:, j] * x[:T - back]
    return y


# ----------------------------------------------------------------------------- mixers (one sequence, positions 0..T-1)
def channel_delta(h, w, m, eps):
    """The gated delta rule whose decay is a vector over a head's key channels, token by token."""
    T, H, G, dk, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = silu(causal_conv(h @ w("q").T, w("q.conv"))).view(T, G, dk)
    k = silu(causal_conv(h @ w("k").T, w("k.conv"))).view(T, G, dk)
    v = silu(causal_conv(h @ w("v").T, w("v.conv"))).view(T, H, dv)
    q, k = unit(q) * dk ** -0.5, unit(k)
    beta = torch.sigmoid(h @ w("b").T)
    rate = softplus((h @ w("a1").T) @ w("a2").T + w("dt_bias")).view(T, H, dk)
    g = torch.exp(-torch.exp(w("A_log"))[:, None] * rate)
    of = [head // (H // G) for head in range(H)]                     # the key head of every head
    o = torch.zeros((T, H, dv), dtype=F)
    S = torch.zeros((H, dk, dv), dtype=F)
    for t in range(T):
        kt, qt = k[t, of], q[t, of]
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, kt))
        S = S + kt[:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hkv,hk->hv", S, qt)
    o = rms_norm(o, w("norm"), eps).reshape(T, H * dv)
    return (o * torch.sigmoid((h @ w("g1").T) @ w("g2").T)) @ w("o").T


def gated_attention(h, w, m, eps, sink=True):
    """Grouped-query softmax attention over every earlier position: biases, a rotation by halves, values over their root
    mean square, one more term exp(sink) in each denominator, and a sigmoid gate per head on the head's result."""
    T, H, G, dk, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rotate_halves((h @ w("q").T + w("q.b")).view(T, H, dk), m["rot"]["dims"], m["rot"]["base"])
    k = rotate_halves((h @ w("k").T + w("k.b")).view(T, G, dk), m["rot"]["dims"], m["rot"]["base"])
    v = rms_norm((h @ w("v").T + w("v.b")).view(T, G, dv), None, eps)
    gate = torch.sigmoid(h @ w("g").T)
    out = torch.zeros((T, H, dv), dtype=F)
    hidden = torch.triu(torch.ones((T, T), dtype=torch.bool), 1)      # [i, j]: position i does not see j > i
    for head in range(H):
        kv = head // (H // G)
        s = ((q[:, head] @ k[:, kv].T) * m["scale"]).masked_fill(hidden, -torch.inf)
        if sink:                                                        # one more column, with no value
            s = torch.cat([s, w("sink")[head].expand(T, 1)], 1)
        out[:, head] = gate[:, head, None] * (torch.softmax(s, -1)[:, :T] @ v[:, kv])
    return out.reshape(T, H * dv) @ w("o").T + w("o.b")


def time_mixing(h, w, m, eps):
    """The recurrence whose inputs each mix the token with the one before it; the current token enters the read-out
    through the bonus u and the state after it."""
    T, H, d = h.shape[0], m["heads"], m["dim"]
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    mix = lambda s: h + (before - h) * w(f"mu.{s}")
    r, k, v = ((mix(s) @ w(s).T).view(T, H, d) for s in "rkv")
    gate = silu(mix("g") @ w("g").T)
    decay = torch.exp(-torch.exp(torch.tanh(mix("w") @ w("w1").T) @ w("w2").T + w("w0"))).view(T, H, d)
    o = torch.zeros((T, H, d), dtype=F)
    S = torch.zeros((H, d, d), dtype=F)
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hkv,hk->hv", S + w("u")[:, :, None] * kv, r[t])
        S = decay[t][:, :, None] * S + kv
    o = rms_norm(o, None, eps).reshape(T, H * d) * w("norm")
    return (o * gate) @ w("o").T


def side_by_side(h, w, m, eps):
    sub = lambda side: (lambda n: w(f"{side}.{n}"))
    left = gated_attention(h, sub("left"), m["left"], eps)
    right = time_mixing(h, sub("right"), m["right"], eps)
    return 0.5 * (rms_norm(left, w("left.out"), eps) + rms_norm(right, w("right.out"), eps))


def latent_of(h, w, eps):
    """What a latent attention layer caches: the normed latent [T, kv_rank]."""
    return rms_norm(h @ w("dkv").T, w("dkv.norm"), eps)


def latent_attention(h, w, m, eps, c):
    """Softmax attention whose queries pass a normed low-rank vector and whose keys and values are made per head from the
    cached latent c."""
    T, H, dk, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (rms_norm(h @ w("dq").T, w("dq.norm"), eps) @ w("uq").T).view(T, H, dk)
    k = (c @ w("uk").T).view(T, H, dk)
    v = (c @ w("uv").T).view(T, H, dv)
    out = torch.zeros((T, H, dv), dtype=F)
    hidden = torch.triu(torch.ones((T, T), dtype=torch.bool), 1)
    for head in range(H):
        s = ((q[:, head] @ k[:, head].T) * m["scale"]).masked_fill(hidden, -torch.inf)
        out[:, head] = torch.softmax(s, -1) @ v[:, head]
    return out.reshape(T, H * dv) @ w("o").T


# ----------------------------------------------------------------------------- feed-forward
def dense(h, w):
    return (silu(h @ w("gate").T) * (h @ w("up").T)) @ w("down").T


def routed_experts(h, w, mlp, forced=None):
    """Each token's `top` experts by sigmoid score; an expert (up, squared relu, down) is applied to its score times the
    input.  forced [T, top]: use these experts instead of choosing.  Returns (result, chosen [T, top])."""
    top = mlp["router"]["top"]
    s = torch.sigmoid(h @ w("router").T)
    chosen = torch.topk(s, top, dim=-1).indices if forced is None else forced.to(torch.long)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in chosen[t].tolist():
            z = w(f"e{e}.up") @ (s[t, e] * h[t])
            out[t] += w(f"e{e}.down") @ torch.clamp(z, min=0) ** 2
    return out, chosen


# ----------------------------------------------------------------------------- the streams
def read_streams(xs, w):
    return sum(w("in")[s] * xs[s] for s in range(len(xs)))


def mix_streams(xs, y, w):
    """Every stream is rebuilt from what the streams before the add give to it (mix[s, t]: stream s to stream t) and the sublayer's result."""
    n = len(xs)
    return [sum(w("mix")[s, t] * xs[s] for s in range(n)) + w("out")[t] * y for t in range(n)]


# ----------------------------------------------------------------------------- the model
def forward(cfg, weights, tokens, forced=None, layers_out=None, mixers=None):
    """Logits [T, vocab] of one sequence.  forced: {layer: [T, top]} experts to use in place of the router's choice.
    forward.chosen holds the experts each routed layer chose.  layers_out: a list that receives the sum of the streams after
    every layer.  mixers: {type: function} used in place of the functions above."""
    W = {k: v.to(F) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    kinds = {"channel_delta": channel_delta, "parallel": side_by_side, "latent_attention": latent_attention, **(mixers or {})}
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    xs = [x.clone() for _ in range(cfg["streams"])]
    cached = {}
    forward.chosen = {}
    for i, L in enumerate(cfg["layers"]):
        m, w = L["mixer"], (lambda n, i=i: W[f"l{i}.mix.{n}"])
        hc = lambda q, i=i: (lambda n: W[f"l{i}.hc{q}.{n}"])
        h = rms_norm(read_streams(xs, hc(1)), W[f"l{i}.norm1"], eps)
        if L["type"] == "latent_attention":
            if m.get("kv_from") is None:
                cached[i] = latent_of(h, w, eps)
            y = kinds[L["type"]](h, w, m, eps, cached[i if m.get("kv_from") is None else m["kv_from"]])
        else:
            y = kinds[L["type"]](h, w, m, eps)
        xs = mix_streams(xs, y, hc(1))
        if L.get("mlp") is not None:
            h = rms_norm(read_streams(xs, hc(2)), W[f"l{i}.norm2"], eps)
            wm = lambda n, i=i: W[f"l{i}.mlp.{n}"]
            if L["mlp"]["kind"] == "dense":
                y = dense(h, wm)
            else:
                y, forward.chosen[i] = routed_experts(h, wm, L["mlp"], None if forced is None else forced.get(i))
            xs = mix_streams(xs, y, hc(2))
        if layers_out is not None:
            layers_out.append(sum(xs))
    return rms_norm(sum(xs), W["final.norm"], eps) @ W["head"].T
