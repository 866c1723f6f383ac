"""The Kodatar decoder in the engine against the plain implementation (tests/plain_kodatar.py): the new kernels alone, each
mechanism alone (models of one layer), whole prompts against token-by-token decoding, portions down to two tokens, mixed
batches with so few pages and slots that both are used again, long decoding, and greedy generation through the engine's
entry point.

Where random weights would hide a fault the inputs are made so that it shows: the score scale of an attention layer is
raised so that the softmax of every (position, head) rests on few keys (a key wrongly seen or hidden, one position off at a
chunk's edge or a page's border, then moves that position's logits by far more than rounding), a model is built whose every
query looks for ONE token (at a chunk's edge, or hundreds of positions back), rotations are scaled within a context of some
tens of positions so that the slowed pairs turn visibly, result rows that nobody may read hold NaN, and a test of the premise
breaks the plain implementation mechanism by mechanism."""
import copy

import pytest
import torch

import helpers
import kodatar_configs as kc
import kodatar_helpers as kh
import plain_kodatar as pk

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]


# ------------------------------------------------------------------------------------------------- kernels alone
@pytest.mark.parametrize("D", [24, 50, 1000, 2052, 4104])
@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
def test_the_norm_between_sublayers_with_routed_rows(D, dt):
    """h += LN(gate y + weighted rows + x_weight x), then the next norm, the stream itself, or picked rows only; a row of
    weight zero holds NaN and must not be read."""
    from quench6k_b200 import ops
    g = torch.Generator().manual_seed(D)
    T, S, eps = 7, 3, 1e-5
    r = lambda *s: torch.randn(*s, generator=g)
    h, wa, ba, w, b, vec = r(T, D), r(D), r(D), r(D), r(D), r(D)
    y, x, xw, gate = r(2, T, D), r(T, D).to(dt), torch.rand(T, generator=g), torch.rand(T, generator=g)
    xw[2] = 0.0
    pw, py, place = torch.rand(T, S, generator=g), r(T * S, D), torch.randperm(T * S, generator=g).to(torch.int32)
    pw[0, 1] = pw[3, 0] = pw[6, 2] = 0.0
    pw[5] = 0.0
    dev = {k: v.cuda() for k, v in dict(h=h, wa=wa, ba=ba, w=w, b=b, y=y, x=x, xw=xw, gate=gate, pw=pw, vec=vec).items()}
    for pair_row in (None, place):
        rows = py[pair_row.view(-1).long()].view(T, S, D) if pair_row is not None else py.view(T, S, D)
        dead = py.clone()
        for t, s in (pw == 0).nonzero().tolist():
            dead[int(pair_row[t * S + s]) if pair_row is not None else t * S + s] = float("nan")
        rows = torch.where(pw[..., None] == 0, torch.zeros(()), rows).double()
        pr = pair_row.view(T, S).contiguous().cuda() if pair_row is not None else None
        for with_y, with_x, with_gate in ((True, True, True), (True, False, True), (False, True, False), (True, True, False)):
            u = (pw.double()[..., None] * rows).sum(1)
            if with_y:
                u = u + (gate.double()[:, None] if with_gate else 1.0) * y.double().sum(0)
            if with_x:
                u = u + xw.double()[:, None] * x.double()
            mix = (dead.cuda(), pr, dev["pw"], dev["x"] if with_x else None, dev["xw"] if with_x else None, dev["gate"] if with_gate else None)
            yy = dev["y"] if with_y else None
            want_h = h.double() + pk.layer_norm(u, wa.double(), ba.double(), eps)
            want = pk.layer_norm(want_h, w.double(), b.double(), eps)
            tol = 1e-4 if dt == torch.float32 else 0.05
            hh = dev["h"].clone()
            out = ops.layernorm(hh, dev["w"], dev["b"], eps, dt, after=(yy, dev["wa"], dev["ba"]), mixture=mix)
            assert (hh.double().cpu() - want_h).abs().max() < 1e-4 and (out.double().cpu() - want).abs().max() < tol
            # the stream itself into the left half of a wider buffer
            hh, buf = dev["h"].clone(), torch.full((T, 2 * D), 7.0, dtype=dt).cuda()
            ops.layernorm(hh, None, None, eps, dt, after=(yy, dev["wa"], dev["ba"]), mixture=mix, raw=buf[:, :D])
            assert torch.equal(buf[:, :D], hh.to(dt)) and bool((buf[:, D:] == 7.0).all()) and (hh.double().cpu() - want_h).abs().max() < 1e-4
            # picked rows (one of them twice): normed as they would stand, the stream untouched
            pick = torch.tensor([6, 2, 2], dtype=torch.int32).cuda()
            hh = dev["h"].clone()
            out = ops.layernorm(hh, dev["w"], dev["b"], eps, dt, rows=pick, after=(yy, dev["wa"], dev["ba"]), mixture=mix)
            assert torch.equal(hh, dev["h"]) and (out.double().cpu() - want[[6, 2, 2]]).abs().max() < tol
            # the stream replaced
            hh = dev["h"].clone()
            out = ops.layernorm(hh, dev["w"], dev["b"], eps, dt, replace=(yy, dev["vec"]), mixture=mix)
            want_h = u + vec.double()
            assert (hh.double().cpu() - want_h).abs().max() < 1e-4
            assert (out.double().cpu() - pk.layer_norm(want_h, w.double(), b.double(), eps)).abs().max() < tol


@pytest.mark.parametrize("E, k, groups, identity, slices", [(9, 3, (3, 2), 3, 1), (8, 4, (2, 1), 0, 2), (12, 5, (4, 2), 11, 1), (5, 5, None, 2, 1),
                                                            (64, 6, (8, 3), 16, 3), (9, 2, (9, 4), 1, 1), (300, 40, (10, 10), 100, 1), (16, 1, (16, 1), 4, 1)])
def test_choice_of_experts(E, k, groups, identity, slices):
    """Softmax scores, a correction that steers the choice, groups by their best value, renormalised weights, the identity
    experts' weights summed beside the others, the gate's column: against the plain implementation, token by token."""
    from quench6k_b200 import ops
    g = torch.Generator().manual_seed(E * k)
    T, N = 70, -(-(E + 1) // 8) * 8
    z = torch.randn(slices, T, N, generator=g) * 2
    corr = torch.randn(E, generator=g) * 0.3                # of the scores' size and of both signs: choice values go negative
    router = {"experts": E - identity, "identity": identity, "top": k}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    sel_e, sel_w, *more = ops.route_biased((z if slices > 1 else z[0]).contiguous().cuda(), k, corr.cuda(), 1.0, groups=groups, scoring="softmax",
                                           group_worth="best", experts=E, identity=identity, gate=True)
    gate = more.pop()
    same = more.pop() if identity else torch.zeros(T)
    total = z[0].clone()
    for s in range(1, slices):
        total += z[s]
    assert (gate.cpu() - torch.sigmoid(total[:, E])).abs().max() < 1e-6
    for t in range(T):
        chosen, wt = pk.choose_experts(total[t, :E].double(), corr.double(), router)
        weight = dict(zip(chosen.tolist(), wt.tolist()))
        assert sorted(sel_e[t].tolist()) == sorted(weight), f"token {t}"
        for e, w in zip(sel_e[t].tolist(), sel_w[t].tolist()):
            assert abs(w - (weight[e] if e < E - identity else 0.0)) < 1e-6
        assert abs(float(same[t]) - sum(w for e, w in weight.items() if e >= E - identity)) < 1e-6


@pytest.mark.parametrize("T, k, E, live, bm", [(37, 3, 10, 7, 16), (1, 4, 6, 1, 16), (300, 4, 24, 20, 32), (5, 2, 1100, 1030, 16)])
def test_the_permutation_leaves_out_experts_without_matrices(T, k, E, live, bm):
    from quench6k_b200 import ops
    g = torch.Generator().manual_seed(T)
    sel = torch.stack([torch.randperm(E, generator=g)[:k] for _ in range(T)]).to(torch.int32)
    if T == 1:
        sel = torch.tensor([[3, 0, 5, 1]], dtype=torch.int32)
    x = torch.randn(T, 16, generator=g)
    offsets, pair_row, row_token, (_, group, row0, n), xs = ops.moe_plan(sel.cuda(), E, bm, x.cuda(), live=live)
    counts = torch.bincount(sel.view(-1).long(), minlength=E)
    assert offsets.tolist() == [0] + counts.cumsum(0).tolist()
    want = [(e, int(counts[:e].sum()) + i) for e in range(live) for i in range(0, int(counts[e]), bm)]
    assert list(zip(group.tolist(), row0.tolist()))[:int(n)] == want and int(n) == len(want)
    for p, e in enumerate(sel.view(-1).tolist()):
        row = int(pair_row.view(-1)[p])
        assert int(offsets[e]) <= row < int(offsets[e + 1]) and int(row_token[row]) == p // k
        if e < live:
            assert torch.equal(xs[row].cpu(), x[p // k])


@pytest.mark.parametrize("D, dt", [(24, torch.float32), (130, torch.bfloat16)])
def test_scaled_embedding_and_its_copies(D, dt):
    from quench6k_b200 import ops
    g = torch.Generator().manual_seed(D)
    table = torch.randn(11, D, generator=g).to(dt)
    toks = torch.tensor([3, -1, 10, 0], dtype=torch.int32)
    want = table[[3, 7, 10, 0]].float() * 2.7
    for copies, wide in ((0, 0), (1, 2 * D), (2, 2 * D)):
        buf = torch.full((4, 2 * D), 5.0, dtype=dt).cuda()
        view = None if copies == 0 else buf[:, -copies * D:]
        h = ops.embed(toks.cuda(), table.cuda(), fed=torch.tensor([7], dtype=torch.int32).cuda(), scale=2.7, copy=view)
        assert torch.allclose(h.cpu(), want, rtol=1e-6)
        for c in range(copies):
            assert torch.equal(view[:, c * D:(c + 1) * D].cpu(), h.cpu().to(dt))
        if copies < 2:
            assert bool((buf[:, :(2 - copies) * D] == 5.0).all())


@pytest.mark.parametrize("Hq, Hkv, hd, ps, chunk", [(32, 4, 128, 16, 100), (8, 2, 64, 8, 37), (6, 2, 128, 16, 129), (16, 1, 64, 32, 1), (4, 4, 128, 4, 150),
                                                    (8, 1, 128, 64, 64), (4, 2, 128, 16, 1000)])
def test_chunks_in_the_fixed_shape_attention_kernels(Hq, Hkv, hd, ps, chunk):
    """The kernels that split the keys (single tokens, a few, portions) and, for heads of 128, the tcgen05 prompt kernel, with a
    mask of chunks: several requests in one launch, portions that begin inside a chunk and cross its edges, tokens at a chunk's
    first and last position; no page that lies before the first chunk of a request's rows is in its table, and every page
    nobody may read holds NaN."""
    from quench6k_b200 import ops
    G = Hq // Hkv
    g = torch.Generator().manual_seed(Hq * 1000 + hd + chunk)
    lens = [700, 150, 333, 64, 4 * chunk if chunk < 200 else 65, 2 * chunk + 1 if chunk < 200 else 66]
    data = [[torch.randn(n, h, hd, generator=g).to(torch.bfloat16) for h in (Hq, Hkv, Hkv)] for n in lens]
    refs = []
    for q, k, v in data:
        pos = torch.arange(q.shape[0])
        seen = (pos[None] <= pos[:, None]) & (pos[None] // chunk == pos[:, None] // chunk)
        kk, vv = (x.double().repeat_interleave(G, 1) for x in (k, v))
        s = torch.einsum("ihd,jhd->hij", q.double(), kk) * 0.2
        refs.append(torch.einsum("hij,jhd->ihd", torch.softmax(s.masked_fill(~seen, float("-inf")), -1), vv))
    for mode in ("single", "few", "portions", "prompt"):
        if mode == "prompt" and not ops.attention_tc_supported(hd, G, ps):
            continue
        few = min(2, max(1, 16 // G)) if G <= 8 else 1
        q_lens = {"single": [1] * 6, "few": [few] * 5 + [1], "portions": [130, 150, 33, 3, min(65, lens[4]), 1], "prompt": [700, 150, 133, 64, lens[4], lens[5]]}[mode]
        starts = [n - ql for n, ql in zip(lens, q_lens)]
        n_pages = sum(-(-n // ps) for n in lens) + 3
        perm = torch.randperm(n_pages, generator=g).tolist()
        kp = torch.full((Hkv, n_pages, ps, hd), float("nan"), dtype=torch.bfloat16)
        vp = kp.clone()
        tables = []
        for r, n in enumerate(lens):
            need = -(-n // ps)
            table = sorted(perm[:need]) if r % 2 == 0 else perm[:need]
            perm = perm[need:]
            first = starts[r] // chunk * chunk // ps                 # the page of the first key any row of the step sees
            for t in range(first * ps, n):
                kp[:, table[t // ps], t % ps], vp[:, table[t // ps], t % ps] = data[r][1][t], data[r][2][t]
            tables.append([-1] * first + table[first:])
        width = max(len(t) for t in tables)
        bt = torch.tensor([t + [-1] * (width - len(t)) for t in tables], dtype=torch.int32).cuda()
        ctx = helpers.make_context(q_lens, starts, [tables])
        q = torch.cat([data[r][0][starts[r]:] for r in range(6)]).contiguous().cuda()
        want = torch.cat([refs[r][starts[r]:] for r in range(6)]).reshape(-1, Hq * hd)
        args = (q, kp.cuda(), vp.cuda(), bt, ctx.req_of_token, ctx.positions)
        if mode == "prompt":
            tok0, ntok, _ = ctx.query_tile_pairs(ops.attention_tc_tile_tokens(G), zigzag=False)
            outs = [ops.attention_tc(*args, tok0, ntok, None, None, scale=0.2, chunk=chunk)]
        else:
            rows = ops.attention_mma_tile_rows(hd, G, max(q_lens))
            tok0, ntok, _ = ctx.query_tiles(rows // G)
            outs = [ops.attention_mma(*args, tok0, ntok, rows, None, None, max_splits=m, min_tiles=1, scale=0.2, chunk=chunk) for m in (1, 4, 64)]
        for out in outs:
            err = (out.double().cpu() - want).abs().max() / want.abs().max()
            assert err <= 1.5e-2, (mode, float(err))
    assert ops.tc_status() == 0


PARTS = {                      # experts, identity, top, groups, expert width, shared width, input width
    "plain": (6, 3, 3, (3, 2), 40, 24, 64), "no_shared": (8, 8, 5, (4, 3), 32, 0, 64), "no_identity": (5, 0, 2, None, 24, 16, 48),
    "mostly_identity": (1, 9, 4, (2, 1), 16, 8, 40), "odd": (3, 2, 2, None, 9, 7, 30), "tensor_cores": (16, 4, 4, (4, 3), 256, 192, 512),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", sorted(PARTS))
def test_the_feed_forward_alone(which, dtype):
    """Steps of one token up to hundreds (pairs straight from the choice, the permutation with row tiles), the sum left to the
    norm, made by the part, and added to a stream: against the plain mixture on the experts the part chose."""
    from quench6k_b200.parts.base import Mixture, Runtime, Tap
    from quench6k_b200.parts.ffn import RoutedExperts
    E, same, top, groups, width, shared, D = PARTS[which]
    g = torch.Generator().manual_seed(E + D)
    part = RoutedExperts(D, E, top, width, scoring="softmax", correction=True, groups=groups, group_worth="best", identity=same,
                         shared_intermediate_size=shared, shared_gate=shared > 0)
    W = {t.name: (torch.randn(t.shape, generator=g) * (0.3 if "correction" in t.name else 2.0 / D ** 0.5)).to(torch.bfloat16) for t in part.tensors()}
    rt = Runtime(torch.device("cuda"), torch.float32 if dtype == "float32" else torch.bfloat16)
    part.bind(lambda n: W[n], rt)
    names = {"router": "gate.weight", "correction": "gate.correction", "shared.sg": "shared_gate.weight", "shared.gate": "shared_experts.gate_proj.weight",
             "shared.up": "shared_experts.up_proj.weight", "shared.down": "shared_experts.down_proj.weight"}

    def w(n):
        if n in names:
            return W[names[n]].double()
        e, kind = n[1:].split(".")
        return W[f"experts.{kind}_proj.weight"][int(e)].double()

    mlp = {"expert": {"ff": width}, "router": {"experts": E, "identity": same, "top": top}}
    if groups is not None:
        mlp["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared:
        mlp["shared"] = {"ff": shared}
    for T in (1, 3, 16, 17, 130):
        x = torch.randn(T, D, generator=g).to(torch.bfloat16)
        ctx = helpers.make_context([T], [0], [[[0]]])
        part.routing_tap = Tap(T)
        xn = x.to(rt.dtype).cuda()
        ctx.takes_mixture = True
        y, rows = part.compute(xn, ctx)
        assert isinstance(rows, Mixture) == bool(same or shared)
        summed = rows.made(y) if isinstance(rows, Mixture) else None
        ctx.takes_mixture = False
        chosen = part.routing_tap.buffers[("experts", 0)][:T].long().cpu()
        want, _ = pk.mixture(x.double(), w, mlp, forced=chosen)
        scale = float(want.abs().max())
        tol = 2e-5 if dtype == "float32" else 2e-2
        # the chosen experts are the best of the part's own logits
        z = part.routing_tap.buffers[("router_logits", 0)][:T].double().cpu()
        assert z.shape[1] == E + same
        for t in range(T):
            own, _ = pk.choose_experts(z[t], w("correction"), mlp["router"])
            c = torch.softmax(z[t], 0) + w("correction")
            assert sorted(own.tolist()) == sorted(chosen[t].tolist()) or float(c[own].sum() - c[chosen[t]].sum()) < 1e-5, f"token {t} of {T}"
        h = torch.ones(T, D).cuda()
        part.forward(xn, ctx, h)
        for got, base in ((summed, 0.0), (h, 1.0)):
            if got is not None:
                assert (got.double().cpu() - base - want).abs().max() / scale < tol, f"{which} {dtype} T={T}"
        y, rows = part.compute(xn, ctx)
        if same or shared:
            assert rows is None and (y.double().cpu() - want).abs().max() / scale < tol


# ------------------------------------------------------------------------------------------------- one mechanism alone
SC = (4.0, 1.0, 3.0, 40)
ONE = {
    "chunk": (kc.attention(4, 2, 16, 24, 0.8, 19, 8, 100.0, SC), None),
    "chunk_of_pages": (kc.attention(2, 1, 16, 8, 0.7, 64, 16, 20.0, SC), None),
    "chunk_of_one": (kc.attention(3, 3, 6, 10, 0.5, 1, 4, 9.0), None),
    "chunk_never_reached": (kc.attention(2, 2, 8, 8, 0.8, 1000, 6, 300.0, (8.0, 1.0, 4.0, 300)), None),
    "chunk_one_key_head": (kc.attention(6, 1, 24, 16, 0.6, 23, 24, 50.0), None),
    "chunk_no_rotation": (kc.attention(2, 2, 10, 7, 0.8, 30, 0, 50.0), None),
    "chunk_tensor_cores": (kc.attention(4, 2, 64, 96, 0.4, 48, 32, 1000.0, (8.0, 1.0, 4.0, 100)), None),
    "chunk_equal_widths": (kc.attention(4, 2, 128, 128, 0.3, 70, 128, 5000.0, (8.0, 1.0, 4.0, 100)), None),
    "experts": (kc.attention(2, 1, 8, 12, 0.6, 23, 8, 20.0, mlp=kc.ff(6, 3, 20, 3, groups=(3, 2), shared=12)), None),
    "experts_all_chosen": (kc.attention(2, 2, 8, 8, 0.6, 11, 8, 20.0, mlp=kc.ff(3, 5, 12, 2)), None),
    "experts_one_chosen": (kc.attention(2, 1, 8, 16, 0.5, 9, 4, 20.0, mlp=kc.ff(2, 1, 20, 4, groups=(2, 1), shared=8)), None),
    "passes": (kc.attention(2, 1, 8, 12, 0.5, 17, 8, 30.0, SC), (0, 1, 4)),
    "one_pass": (kc.attention(3, 3, 8, 8, 0.5, 26, 8, 30.0, mlp=kc.ff(4, 2, 16, 2, shared=12)), (0, 1, 1)),
    "passes_tensor_cores": (kc.attention(2, 1, 64, 64, 0.3, 37, 64, 300.0, mlp=kc.ff(6, 2, 64, 2, groups=(2, 1), shared=64)), (0, 1, 2)),
}


def _is_tc(name):
    return name.endswith(("tensor_cores", "equal_widths"))


@pytest.fixture(scope="module", params=sorted(ONE))
def single(request, tmp_path_factory):
    name = request.param
    layer, loop = ONE[name]
    folder = str(tmp_path_factory.mktemp(name))
    cfg = kc.one_layer(layer, width=128 if _is_tc(name) else 48, page=16 if _is_tc(name) else 4, loop=loop)
    cfg, weights = kh.make_folder(folder, cfg, seed=3, init_std=0.3, doctor=kh.lively)
    reqs = {"long": helpers.random_tokens(330, cfg["vocab"], 1), "short": helpers.random_tokens(9, cfg["vocab"], 2),
            "one": helpers.random_tokens(1, cfg["vocab"], 3)}
    return name, folder, cfg, weights, reqs


@pytest.mark.parametrize("dtype", DTYPES)
def test_mechanism_alone_whole_prompt(single, dtype):
    name, folder, cfg, weights, reqs = single
    steps, mt = helpers.schedule_whole(reqs)
    kh.replay_and_compare(folder, cfg, weights, reqs, steps, mt, dtype, f"{name} whole")


@pytest.mark.parametrize("dtype", DTYPES)
def test_mechanism_alone_token_by_token(single, dtype):
    """Every token decoded alone from the first one on: each key is found through the cache of its pass."""
    name, folder, cfg, weights, reqs = single
    reqs = {"long": reqs["long"][:150], "short": reqs["short"]}
    steps, mt = helpers.schedule_tail(reqs, tail=10 ** 6)
    kh.replay_and_compare(folder, cfg, weights, reqs, steps, mt, dtype, f"{name} decoded")


@pytest.mark.parametrize("dtype", DTYPES)
def test_mechanism_alone_portions(single, dtype):
    name, folder, cfg, weights, reqs = single
    for seed in (0, 1):
        steps, mt = helpers.schedule_portions(reqs, seed=seed)
        kh.replay_and_compare(folder, cfg, weights, reqs, steps, mt, dtype, f"{name} portions")


def test_a_fault_would_show(single):
    """The premise of the tests above: each mechanism left out or moved by one is far beyond the tolerance: the plain
    implementation, broken on purpose, differs from itself."""
    name, folder, cfg, weights, reqs = single
    toks = reqs["long"][:150]
    want = kh.plain(cfg, weights, toks)

    def shows(other, what, share=0.15, w=weights, **kw):
        b = pk.forward(other, w, toks, **kw)
        moved = (want - b).abs().max(-1).values / want.abs().max() > 3 * kh.TOL["bfloat16"]
        assert moved.float().mean() > share, f"{name}: {what} does not show ({float(moved.float().mean()):.2f})"

    def changed(change):
        other = copy.deepcopy(cfg)
        change(other)
        return other

    m = cfg["layers"][0]["mixer"]
    if 1 < m["mask"]["size"] < 32 and name.startswith("chunk"):
        shows(changed(lambda c: c["layers"][0]["mixer"]["mask"].update(size=m["mask"]["size"] + 1)), "a chunk one position longer")
    if m["rot"].get("scaling") and name.startswith("chunk") and m["mask"]["size"] > 16:
        shows(changed(lambda c: c["layers"][0]["mixer"]["rot"].pop("scaling")), "a rotation without scaled frequencies")
    shows(changed(lambda c: c.update(logit_scale=2 * c["logit_scale"])), "another scale of the logits", 0.9)
    shows(changed(lambda c: c["embedding"].update(scale=2 * c["embedding"]["scale"])), "another scale of the embedding", 0.2)
    if cfg["layers"][0]["mlp"] is not None:
        if cfg["layers"][0]["mlp"]["router"].get("identity"):
            shows(cfg, "identity experts that answer nothing", 0.05, ffn=lambda *a: pk.mixture(*a, identity=0.0))
        if cfg["layers"][0]["mlp"].get("shared"):
            shows(cfg, "a shared expert with another gate", 0.1, w={**weights, "l0.mlp.shared.sg": weights["l0.mlp.shared.sg"] * -1})
        if name != "experts_all_chosen":
            shows(cfg, "a choice without the correction", 0.05, w={**weights, "l0.mlp.correction": weights["l0.mlp.correction"] * 0})
    if "loop" in cfg:
        D = cfg["width"]
        half = weights["loop.in"].clone()
        half[:, D:] = 0
        shows(cfg, "passes without the embedding output", w={**weights, "loop.in": half})
        shows(cfg, "passes without their vectors", w={**weights, "loop.step": weights["loop.step"] * 0})
        shows(changed(lambda c: c["loop"].update(times=1)) if cfg["loop"]["times"] > 1 else changed(lambda c: c.pop("loop")), "another number of passes")
        if cfg["loop"]["times"] > 1:
            shows(cfg, "passes in another order", w={**weights, "loop.step": weights["loop.step"].flip(0)})


# ------------------------------------------------------------------------------------------------- a key that stands out
BEACON = 17


def _beacon_tokens(n, vocab, seed):
    return [t if t != BEACON else 3 for t in helpers.random_tokens(n, vocab, seed)]


def _beacon(layers, heads, kv_heads, dim, vdim, width, looped):
    """Channel 0 of every layer's input is one (its norm says so) and channel 1 is large for one token and near zero for all
    others.  The last entry of every key head reads channel 1 and the last entry of every query head reads channel 0: every
    query looks, above all, for that one token, and the entry lies outside the part of the head that turns.  The first value
    entry tells the token from the others.  No sublayer's result, and no entry of a pass, changes channel 1."""
    def doctor(w):
        w["embed"][:, 1] = 0.0
        w["embed"][BEACON, 1] = 3.0
        w["final.norm"][1] = w["final.norm.b"][1] = 0.0
        if looped:
            w["loop.in"][1] = 0.0
            w["loop.in"][1, width + 1] = 1.0
            w["loop.step"][:, 1] = 0.0
        for i in range(layers):
            L = f"l{i}."
            w[L + "norm1"][0], w[L + "norm1.b"][0] = 0.0, 1.0
            w[L + "norm1"][1], w[L + "norm1.b"][1] = 1.0, 0.0
            w[L + "norm1b"][1] = w[L + "norm1b.b"][1] = 0.0
            w[L + "mix.q.norm"][dim - 1] = w[L + "mix.k.norm"][dim - 1] = 1.0
            for h in range(kv_heads):
                w[L + "mix.k"][h * dim + dim - 1] = 0.0
                w[L + "mix.k"][h * dim + dim - 1, 1] = 10.0
                w[L + "mix.v"][h * vdim] = 0.0
                w[L + "mix.v"][h * vdim, 1] = 3.0
            for h in range(heads):
                w[L + "mix.q"][h * dim + dim - 1] = 0.0
                w[L + "mix.q"][h * dim + dim - 1, 0] = 6.0
    return doctor


def _beacon_model(folder, layer, n_layers, loop, seed):
    m = layer["mixer"]
    cfg = kc.model([layer] * n_layers, width=48, vocab=61, page=4, loop=loop)
    return kh.make_folder(folder, cfg, seed=seed, init_std=0.15, doctor=_beacon(n_layers, m["heads"], m["kv_heads"], m["dim"], m["vdim"], 48, loop is not None))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, kv_heads, dim, vdim, size, loop", [(2, 1, 8, 5, 13, None), (4, 2, 8, 10, 50, (0, 1, 2)), (3, 3, 16, 16, 32, (1, 2, 2))])
def test_a_key_at_the_edge_of_a_chunk(tmp_path, heads, kv_heads, dim, vdim, size, loop, dtype):
    """Two layers, or one of them in two passes (each with a cache of its own).  The token every query looks for stands such
    that the chunk's last position rests on it and the next chunk's first does not, in prompts (whole and in portions) and
    among tokens decoded one by one."""
    layer = kc.attention(heads, kv_heads, dim, vdim, 1.2, size, 4, 100.0, (4.0, 1.0, 3.0, 40))
    cfg, weights = _beacon_model(str(tmp_path), layer, 2, loop, 11)
    toks = _beacon_tokens(max(230, 5 * size + 20), cfg["vocab"], 5)
    # places that a chunk one position shorter hides from the chunk's last position and that a chunk one position longer
    # shows to the next chunk's first
    places = (size + 3, 4 * (size + 1) + 1)
    for p in places:
        toks[p] = BEACON
    reqs = {"b": toks}
    want = kh.plain(cfg, weights, toks)
    scale = float(want.abs().max())
    narrower, wider = copy.deepcopy(cfg), copy.deepcopy(cfg)
    for L in narrower["layers"]:
        L["mixer"]["mask"]["size"] = size - 1
    for L in wider["layers"]:
        L["mixer"]["mask"]["size"] = size + 1
    less, more = kh.plain(narrower, weights, toks), kh.plain(wider, weights, toks)
    edges = []
    for p in places:
        last = p // size * size + size - 1                    # the last position that sees the token
        gone = last + 1
        assert float((want[last] - less[last]).abs().max()) > 0.1 * scale, "the last position that sees the token does not rest on it"
        assert float((want[gone] - more[gone]).abs().max()) > 0.1 * scale, "the first position beyond the token would not rest on it"
        edges += [last, gone]
    for what, (steps, mt) in {"whole": helpers.schedule_whole(reqs), "decoded": helpers.schedule_tail(reqs, tail=130),
                              "from the start": helpers.schedule_tail(reqs, tail=10 ** 6), "portions": helpers.schedule_portions(reqs, seed=2),
                              "portions again": helpers.schedule_portions(reqs, seed=3)}.items():
        outputs, _ = helpers.run_replay(str(tmp_path), dtype, steps, mt, max_requests=2)
        got = helpers.collect(reqs, steps, outputs)["b"]
        kh.assert_close(got, want, dtype, f"edge, {what}")
        for at in edges:                              # the edges themselves, held to the plain tolerance whatever the rest does
            err = float((got[at].double() - want[at]).abs().max()) / scale
            assert err <= kh.TOL[dtype], f"edge, {what} {dtype}: position {at}: {err:.3e}"


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_key_far_away(tmp_path, dtype):
    """A chunk of several hundred positions: the token every query looks for stands near the start, and positions hundreds of
    tokens on (in the prompt, in portions and decoded) still rest on it, in every pass."""
    cfg, weights = _beacon_model(str(tmp_path), kc.attention(2, 1, 8, 5, 1.5, 500, 4, 100.0, (4.0, 1.0, 3.0, 40)), 1, (0, 1, 2), 12)
    toks = _beacon_tokens(390, cfg["vocab"], 6)
    toks[5] = BEACON
    reqs = {"f": toks}
    want = kh.plain(cfg, weights, toks)
    without = list(toks)
    without[5] = 3
    other = kh.plain(cfg, weights, without)
    assert float((want[300:] - other[300:]).abs().max(-1).values.min()) > 0.05 * float(want.abs().max()), "positions hundreds of tokens on do not rest on the token"
    for what, (steps, mt) in {"whole": helpers.schedule_whole(reqs), "decoded": helpers.schedule_tail(reqs, tail=60),
                              "portions": helpers.schedule_portions(reqs, seed=4)}.items():
        outputs, _ = helpers.run_replay(str(tmp_path), dtype, steps, mt, max_requests=2)
        kh.assert_close(helpers.collect(reqs, steps, outputs)["f"], want, dtype, f"far key, {what}")


# ------------------------------------------------------------------------------------------------- whole models
LENGTHS = {"K1": [71, 130, 45, 96, 64, 33, 1, 58, 77], "K2": [85, 140, 37, 101, 2, 50, 90, 125, 44], "K3": [90, 217, 129, 48, 75, 40, 150, 66, 83],
           "K4": [70, 33, 131, 20, 64, 3, 95, 41, 58]}


@pytest.fixture(scope="module", params=sorted(LENGTHS))
def model(request, tmp_path_factory):
    name = request.param
    folder = str(tmp_path_factory.mktemp(name))
    cfg, weights = kh.make_folder(folder, kc.get(name), seed=7, init_std=0.12, doctor=kh.lively)
    reqs = {f"r{i}": helpers.random_tokens(n, cfg["vocab"], 100 + i) for i, n in enumerate(LENGTHS[name])}
    return {"name": name, "folder": folder, "cfg": cfg, "weights": weights, "requests": reqs}


@pytest.mark.parametrize("dtype", DTYPES)
def test_model_whole(model, dtype):
    steps, mt = helpers.schedule_whole(model["requests"])
    kh.replay_and_compare(model["folder"], model["cfg"], model["weights"], model["requests"], steps, mt, dtype, model["name"] + " whole")


def test_the_stream_after_every_layer(model):
    """The residual stream after each executed layer against the plain implementation's, float32: a layer that is wrong is named."""
    import quench6k_b200 as q
    toks = model["requests"]["r0"]
    want = []
    pk.forward(model["cfg"], model["weights"], toks, layers_out=want)
    runner = q.engine.ModelRunner.from_folder(model["folder"], dtype="float32", page_size=model["cfg"]["kv_page_size"], num_pages=64, max_requests=2)
    got = kh.streams_of(runner, toks)
    assert len(got) == len(want)
    for i, (a, b) in enumerate(zip(got, want)):
        err = float((a.double().cpu() - b).abs().max() / b.abs().max())
        assert err < 1e-4, f"{model['name']}: the stream after executed layer {i}: {err:.3e}"


@pytest.mark.parametrize("dtype", DTYPES)
def test_model_prefill_then_decode(model, dtype):
    steps, mt = helpers.schedule_tail(model["requests"], tail=40)
    kh.replay_and_compare(model["folder"], model["cfg"], model["weights"], model["requests"], steps, mt, dtype, model["name"] + " tail")


@pytest.mark.parametrize("dtype", DTYPES)
def test_model_portions(model, dtype):
    steps, mt = helpers.schedule_portions(model["requests"], seed=5)
    kh.replay_and_compare(model["folder"], model["cfg"], model["weights"], model["requests"], steps, mt, dtype, model["name"] + " portions")


@pytest.mark.parametrize("dtype", DTYPES)
def test_model_mixed_batches_reuse_pages_and_slots(model, dtype):
    """Up to four live requests, unequal portions beside single tokens, requests that sit steps out; nine requests go
    through four slots and a pool of the live requests' size, so every slot and most pages are used again."""
    page = model["cfg"]["kv_page_size"]
    for seed in (0, 1):
        steps, mt = helpers.schedule_mixed(model["requests"], page, seed=seed, max_live=4)
        got = kh.replay_and_compare(model["folder"], model["cfg"], model["weights"], model["requests"], steps, mt, dtype,
                                    model["name"] + " mixed", max_requests=4)
    if dtype == "float32":
        # and the same requests each alone: what else is in the batch, and which pages and slots are used, changes nothing
        steps, mt = helpers.schedule_whole(model["requests"])
        outputs, _ = helpers.run_replay(model["folder"], dtype, steps, mt)
        alone = helpers.collect(model["requests"], steps, outputs)
        for rid in model["requests"]:
            kh.assert_close(got[rid], alone[rid], dtype, f"{model['name']} {dtype} {rid} batched against alone", tol=2e-5)


@pytest.mark.parametrize("dtype", DTYPES)
def test_model_many_decoding_together(model, dtype):
    page = model["cfg"]["kv_page_size"]
    reqs = {rid: t for rid, t in model["requests"].items() if len(t) > 12}
    steps, mt = helpers.schedule_wide_decode(reqs, page)
    kh.replay_and_compare(model["folder"], model["cfg"], model["weights"], reqs, steps, mt, dtype, model["name"] + " wide decode",
                          max_requests=len(reqs))


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(model, dtype):
    """A short prompt and hundreds of tokens decoded one by one: chunks and pages pass over decoded tokens, the decode steps
    are replayed from a recorded graph."""
    reqs = {"d": helpers.random_tokens(420, model["cfg"]["vocab"], 9)}
    steps, mt = helpers.schedule_tail(reqs, tail=410)
    kh.replay_and_compare(model["folder"], model["cfg"], model["weights"], reqs, steps, mt, dtype, model["name"] + " long decode")


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_long_prompt(model, dtype):
    """A prompt of 1,100 tokens whole, in portions, and with its last tokens decoded: chunks many times over."""
    if model["name"] != "K1":
        pytest.skip("one of the models is enough for the length (the plain implementation is slow)")
    reqs = {"p": helpers.random_tokens(1100, model["cfg"]["vocab"], 21)}
    for what, (steps, mt) in {"whole": helpers.schedule_whole(reqs), "portions": helpers.schedule_portions(reqs, seed=8),
                              "tail": helpers.schedule_tail(reqs, tail=40)}.items():
        kh.replay_and_compare(model["folder"], model["cfg"], model["weights"], reqs, steps, mt, dtype, f"{model['name']} long prompt {what}")


def test_greedy_generation_through_the_engine(model):
    """Engine.generate (scheduler, continuous batching, device-side argmax, tokens that stay on the device for the next step,
    CUDA graphs) against greedy decoding with the plain implementation, float32; prompts of unequal length in one engine
    with few pages."""
    import quench6k_b200 as q
    cfg, weights = model["cfg"], model["weights"]
    prompts = [helpers.random_tokens(n, cfg["vocab"], 50 + n) for n in (5, 23, 1, 40, 12, 31)]
    page = cfg["kv_page_size"]
    widest = max(L["mixer"]["mask"]["size"] for L in cfg["layers"])           # a pool must hold the widest chunk
    eng = q.Engine.from_folder(model["folder"], dtype="float32", page_size=page, num_pages=max(4 * (64 // page + 2), widest // page + 3), max_requests=4,
                               max_batch_tokens=32)
    outs = eng.generate(prompts, q.SamplingParams(max_tokens=12, temperature=0))
    for prompt, out in zip(prompts, outs):
        toks = list(prompt)
        for i in range(12):
            logits = kh.plain(cfg, weights, toks)[-1]
            top2 = logits.topk(2).values
            if float(top2[0] - top2[1]) < 1e-3 * float(logits.abs().max()):
                break                                  # a near-tie: float32 may pick either; the continuation is not comparable
            assert out.tokens[i] == int(logits.argmax()), f"{model['name']}: prompt of {len(prompt)}, generated token {i}"
            toks.append(out.tokens[i])
    eng.runner.manager.check()


def test_command_line_generates(model):
    """`generate` of the command line on a Kodatar model folder: the model class comes from config.json."""
    import os
    import subprocess
    import sys
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg, weights = model["cfg"], model["weights"]
    prompt = helpers.random_tokens(11, cfg["vocab"], 77)
    r = subprocess.run([sys.executable, "-m", "quench6k_b200", "generate", "--model", model["folder"], "--prompt-ids", ",".join(map(str, prompt)),
                        "--n", "6", "--dtype", "float32", "--context", "512"], cwd=root, capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    toks = list(prompt)
    for _ in range(6):
        logits = kh.plain(cfg, weights, toks)[-1]
        top2 = logits.topk(2).values
        if float(top2[0] - top2[1]) < 1e-3 * float(logits.abs().max()):
            return
        toks.append(int(logits.argmax()))
    assert "prompt: 11 tokens" in r.stdout and f"ids: {toks[11:]}" in r.stdout
