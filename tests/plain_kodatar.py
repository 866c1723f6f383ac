"""A plain, slow implementation of the Kodatar decoder from its equations: one function per mechanism, whole sequences
at a time, double precision, loops where a loop is the clearest way to say it.  It shares nothing with the engine (no
part, no kernel, no cache): the tests compare the engine with it.

A model is (config dict, {tensor name: torch tensor}).  Tensor names: `embed`, `final.norm[.b]`, `loop.in`, `loop.step`, and
per layer i `l<i>.norm1[.b]`, `l<i>.norm1b[.b]`, `l<i>.norm2[.b]`, `l<i>.norm2b[.b]`, `l<i>.mix.*`, `l<i>.mlp.*`.
"""
import math

import torch

F = torch.float64


# ----------------------------------------------------------------------------- small pieces
def layer_norm(x, w, b, eps):
    mu = x.mean(-1, keepdim=True)
    var = ((x - mu) ** 2).mean(-1, keepdim=True)
    return (x - mu) / torch.sqrt(var + eps) * w + b


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def frequencies(rot):
    """The angle per position of every rotating pair.  Pairs that turn slowly (few turns within the original context) are
    slowed by `factor`, pairs that turn fast keep their pace, those between are blended linearly in the number of turns."""
    out = []
    scaling = rot.get("scaling")
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        if scaling is not None:
            wavelength = 2.0 * math.pi / f
            turns = scaling["original"] / wavelength
            if turns < scaling["low"]:
                f = f / scaling["factor"]
            elif turns <= scaling["high"]:
                keep = (turns - scaling["low"]) / (scaling["high"] - scaling["low"]) if scaling["high"] > scaling["low"] else 1.0
                f = (1.0 - keep) * f / scaling["factor"] + keep * f
        out.append(f)
    return out


def rotate_halves(x, positions, rot):
    """x [T, heads, n]: the first `dims` entries of the last axis turn; entry i pairs with entry i + dims/2."""
    out = x.clone()
    half = rot["dims"] // 2
    for i, f in enumerate(frequencies(rot)):
        ang = positions.to(F) * f
        c, s = torch.cos(ang)[:, None], torch.sin(ang)[:, None]
        out[..., i] = x[..., i] * c - x[..., i + half] * s
        out[..., i + half] = x[..., i + half] * c + x[..., i] * s
    return out


# ----------------------------------------------------------------------------- the mixer (one sequence, positions 0..T-1)
def chunked_attention(h, w, m, eps):
    """Grouped-query attention inside chunks of `mask.size` positions counted from position 0: q and k normed per head, then
    rotated; values of their own width."""
    T = h.shape[0]
    H, G, d, dv, C = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["mask"]["size"]
    pos = torch.arange(T)
    q = rotate_halves(rms_norm((h @ w("q").T).view(T, H, d), w("q.norm"), eps), pos, m["rot"])
    k = rotate_halves(rms_norm((h @ w("k").T).view(T, G, d), w("k.norm"), eps), pos, m["rot"])
    v = (h @ w("v").T).view(T, G, dv)
    seen = (pos[None, :] <= pos[:, None]) & (pos[None, :] // C == pos[:, None] // C)
    out = torch.zeros((T, H, dv), dtype=F)
    for head in range(H):
        g = head // (H // G)
        s = (q[:, head] @ k[:, g].T) * m["scale"]
        out[:, head] = torch.softmax(s.masked_fill(~seen, -math.inf), dim=-1) @ v[:, g]
    return out.reshape(T, H * dv) @ w("o").T


# ----------------------------------------------------------------------------- feed-forward
def expert(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def choose_experts(z, correction, router):
    """z [E] router logits of one token (identity experts last) -> (chosen experts, their weights).  The choice goes by
    softmax(z) + correction among the experts of the groups whose largest such value is largest; the weights are the
    softmax scores, divided by their sum."""
    E, top = z.shape[0], router["top"]
    s = torch.softmax(z, dim=0)
    c = s + correction
    groups = router.get("groups")
    if groups is not None and groups["count"] > 1:
        n = E // groups["count"]
        worth = torch.stack([c[g * n:(g + 1) * n].max() for g in range(groups["count"])])
        masked = torch.full_like(c, -math.inf)
        for g in torch.topk(worth, groups["keep"]).indices.tolist():
            masked[g * n:(g + 1) * n] = c[g * n:(g + 1) * n]
        c = masked
    chosen = torch.topk(c, top).indices
    return chosen, weights_of(z, chosen)


def weights_of(z, chosen):
    """The weights of given experts of one token: their softmax scores over all experts, divided by their sum."""
    s = torch.softmax(z, dim=0)[chosen]
    return s / (s.sum() + 1e-20)


def mixture(h, w, mlp, forced=None, identity=1.0):
    """Each token's chosen experts, weighted; an identity expert answers its input; plus the shared expert times one sigmoid
    number per token.  forced [T, top]: use these experts instead of choosing.  identity: what an identity expert multiplies its
    input by (tests that break it on purpose).  Returns (result, chosen [T, top])."""
    z = h @ w("router").T
    out = torch.zeros_like(h)
    all_chosen = []
    for t in range(h.shape[0]):
        chosen, wt = choose_experts(z[t], w("correction"), mlp["router"])
        if forced is not None:
            chosen = forced[t].to(torch.long)
            wt = weights_of(z[t], chosen)
        all_chosen.append(chosen)
        for s in range(chosen.numel()):
            e = int(chosen[s])
            answer = identity * h[t] if e >= mlp["router"]["experts"] else expert(h[t], w(f"e{e}.gate"), w(f"e{e}.up"), w(f"e{e}.down"))
            out[t] = out[t] + wt[s] * answer
    if mlp.get("shared") is not None:
        out = out + torch.sigmoid(h @ w("shared.sg").T) * expert(h, w("shared.gate"), w("shared.up"), w("shared.down"))
    return out, torch.stack(all_chosen)


# ----------------------------------------------------------------------------- the model
def executed_layers(cfg):
    """[(layer index, number of the pass this position opens or None)] in the order they run."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if loop is None:
        return [(i, None) for i in range(n)]
    out = [(i, None) for i in range(loop["start"])]
    for r in range(loop["times"]):
        out += [(i, r if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return out + [(i, None) for i in range(loop["stop"], n)]


def open_pass(x, x0, w_in, step):
    """The stream at the start of a pass: the stream and the embedding output through one matrix, plus the pass's vector."""
    return torch.cat([x, x0], dim=-1) @ w_in.T + step


def forward(cfg, weights, tokens, forced=None, layers_out=None, mixer=chunked_attention, ffn=mixture):
    """Logits [T, vocab] of one sequence.  forced: {executed position: [T, top]} experts to use in place of the router's
    choice.  forward.chosen holds the experts each routed position chose.  layers_out: a list that receives the stream
    after every executed layer.  mixer, ffn: other functions for the mixer and the feed-forward (tests that break them on
    purpose)."""
    W = {k: v.to(F) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    tok = torch.as_tensor(tokens, dtype=torch.long)
    x0 = W["embed"][tok] * cfg["embedding"]["scale"]
    x = x0
    forward.chosen = {}

    def norm(name, y):
        return layer_norm(y, W[name], W[name + ".b"], eps)

    for p, (i, opens) in enumerate(executed_layers(cfg)):
        L = cfg["layers"][i]
        if opens is not None:
            x = open_pass(x, x0, W["loop.in"], W["loop.step"][opens])
        x = x + norm(f"l{i}.norm1b", mixer(norm(f"l{i}.norm1", x), lambda n, i=i: W[f"l{i}.mix.{n}"], L["mixer"], eps))
        if L.get("mlp") is not None:
            f, forward.chosen[p] = ffn(norm(f"l{i}.norm2", x), lambda n, i=i: W[f"l{i}.mlp.{n}"], L["mlp"], None if forced is None else forced.get(p))
            x = x + norm(f"l{i}.norm2b", f)
        if layers_out is not None:
            layers_out.append(x.clone())
    return norm("final.norm", x) @ W["embed"].T * cfg["logit_scale"]
