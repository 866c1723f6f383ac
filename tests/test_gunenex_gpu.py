"""The Gunenex decoder in the engine against the plain implementation (tests/plain_gunenex.py): the new kernels alone,
each mechanism alone (models of one or two layers), whole prompts against token-by-token decoding, portions down to two
tokens, mixed batches with so few pages and slots that both are used again, keys far away and at page borders, long
decoding, and greedy generation through the engine's entry point.

Where random weights would hide a fault the inputs are made so that it shows: decays run from channels that forget at
once to channels that keep everything (gunenex_helpers.spread), score scales are raised so that the softmax of every
(position, head) rests on few keys, and a model is built whose every query looks for ONE token, placed at the start, on
both sides of a page border and inside a page, hundreds of positions back."""
import copy

import pytest
import torch

import gunenex_configs as gc
import gunenex_helpers as gh
import helpers
import plain_gunenex as pg

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]
F = torch.float64


def _portions(lens, cuts, slots):
    """(live requests, step context with their slots, start of each live request's rows) for every step of `cuts`."""
    at = [0] * len(lens)
    for step in range(max(len(c) for c in cuts)):
        live = [i for i in range(len(lens)) if step < len(cuts[i])]
        ctx = helpers.make_context([cuts[i][step] for i in live], [at[i] for i in live], [[[0]] * len(live)])
        ctx.slot_ids = torch.tensor([slots[i] for i in live], dtype=torch.int32).cuda()
        yield live, ctx, {i: (at[i], at[i] + cuts[i][step]) for i in live}
        for i in live:
            at[i] += cuts[i][step]


CUTS = ([[60], [17]], [[1, 1, 1, 2, 29, 1, 25], [1, 1, 13, 2]], [[40, 3, 17], [1, 1, 15]], [[4, 5, 6, 7, 20, 18], [2, 2, 2, 11]])


# ------------------------------------------------------------------------------------------------- kernels alone
@pytest.mark.parametrize("H, G, dk, dv", [(4, 2, 16, 24), (2, 1, 100, 20), (5, 5, 7, 9), (1, 1, 136, 33), (4, 2, 32, 80), (2, 2, 250, 16), (3, 1, 64, 40)])
def test_delta_channel_kernels_in_portions(H, G, dk, dv):
    """Unit vectors, decays per key channel (from exp(-300) to one), the recurrence: over two requests whole and cut into
    portions, with and without the kernel that prepares a step's inputs, against loops in double precision."""
    from quench6k_b200 import ops
    g = torch.Generator().manual_seed(H * dk + dv)
    lens, C = [60, 17], 2 * G * dk + H * dv
    us = [torch.randn(n, C, generator=g) for n in lens]
    ps = [torch.randn(n, H + 3, generator=g) for n in lens]
    decays = [torch.randn(n, H * dk + 2, generator=g) for n in lens]
    A_log, dt_bias = torch.randn(H, generator=g), torch.linspace(-9.0, 30.0, H * dk)[torch.randperm(H * dk, generator=g)]
    want = []
    for u, p, a in zip(us, ps, decays):
        u, p, a = u.double(), p.double(), a.double()
        n = u.shape[0]
        q, k, v = u[:, :G * dk].view(n, G, dk), u[:, G * dk:2 * G * dk].view(n, G, dk), u[:, 2 * G * dk:].view(n, H, dv)
        q, k = pg.unit(q) * dk ** -0.5, pg.unit(k)
        beta = torch.sigmoid(p[:, 2:2 + H])
        dec = torch.exp(-torch.exp(A_log.double())[:, None] * pg.softplus(a[:, 1:1 + H * dk] + dt_bias.double()).view(n, H, dk))
        o = torch.zeros(n, H, dv, dtype=F)
        for h in range(H):
            S = torch.zeros(dk, dv, dtype=F)
            for t in range(n):
                S = dec[t, h][:, None] * S
                S = S + torch.outer(k[t, h // (H // G)], beta[t, h] * (v[t, h] - S.T @ k[t, h // (H // G)]))
                o[t, h] = S.T @ q[t, h // (H // G)]
        want.append(o.view(n, H * dv))
    for prepare in (False, True):
        for cuts in CUTS:
            state = torch.zeros(4, H, dv, dk).cuda()
            state[1] = 7.0
            got = [[], []]
            for live, ctx, span in _portions(lens, cuts, [3, 0]):
                cat = lambda xs: torch.cat([xs[i][span[i][0]:span[i][1]] for i in live]).contiguous().cuda()
                o = ops.delta_channel(cat(us), cat(ps), 2, cat(decays), 1, A_log.cuda(), dt_bias.cuda(), state, ctx.req_of_token, ctx.q_start,
                                      ctx.slot_ids, ctx.R, H, G, dk, dv, prepare=prepare, single=not prepare and ctx.max_q_len == 1)
                row = 0
                for i in live:
                    n = span[i][1] - span[i][0]
                    got[i].append(o[row:row + n].double().cpu())
                    row += n
            for i in (0, 1):
                err = (torch.cat(got[i]) - want[i]).abs().max() / want[i].abs().max()
                assert err < 1e-5, f"prepare {prepare}, cuts {cuts}, request {i}: {float(err):.3e}"
            assert bool((state[1] == 7.0).all()) and bool((state[2] == 0).all())


@pytest.mark.parametrize("H, d, D", [(3, 16, 40), (2, 100, 24), (5, 7, 33), (1, 136, 8), (4, 64, 64)])
def test_time_mixing_kernels_in_portions(H, d, D):
    """The five mixes with the row before (kept in the slot between portions), the bonus, the decays and the recurrence."""
    from quench6k_b200 import ops
    g = torch.Generator().manual_seed(H * d)
    lens = [60, 17]
    xs = [torch.randn(n, D, generator=g) for n in lens]
    mu = torch.randn(5, D, generator=g)
    W = [torch.randn(H * d, D, generator=g) * 0.2 for _ in range(4)]        # r, k, v, w as functions of their mixes
    w0, u = torch.linspace(-9.0, 2.0, H * d)[torch.randperm(H * d, generator=g)].view(H, d), torch.randn(H, d, generator=g)
    want = []
    for x in xs:
        x = x.double()
        n = x.shape[0]
        before = torch.cat([torch.zeros_like(x[:1]), x[:-1]])
        r, k, v, z = ((x + (before - x) * mu[j].double()) @ W[j].double().T for j in range(4))
        r, k, v, dec = r.view(n, H, d), k.view(n, H, d), v.view(n, H, d), torch.exp(-torch.exp(z.view(n, H, d) + w0.double()))
        o, S = torch.zeros(n, H, d, dtype=F), torch.zeros(H, d, d, dtype=F)
        for t in range(n):
            kv = k[t][:, :, None] * v[t][:, None, :]
            o[t] = ((S + u.double()[:, :, None] * kv) * r[t][:, :, None]).sum(1)
            S = dec[t][:, :, None] * S + kv
        want.append(o.view(n, H * d))
    for cuts in CUTS:
        state, prev = torch.zeros(4, H, d, d).cuda(), torch.zeros(4, D).cuda()
        state[1], prev[1] = 7.0, 5.0
        got = [[], []]
        for live, ctx, span in _portions(lens, cuts, [3, 0]):
            x = torch.cat([xs[i][span[i][0]:span[i][1]] for i in live]).contiguous().cuda()
            m = ops.token_shift(x, mu.cuda(), prev, ctx.req_of_token, ctx.q_start, ctx.slot_ids)
            r, k, v, z = (torch.mm(m[j], W[j].cuda().T).contiguous() for j in range(4))
            o = ops.time_mix(r, k, v, z, w0.cuda(), u.cuda(), state, ctx.q_start, ctx.slot_ids, ctx.R)
            row = 0
            for i in live:
                n = span[i][1] - span[i][0]
                got[i].append(o[row:row + n].double().cpu())
                row += n
        for i in (0, 1):
            err = (torch.cat(got[i]) - want[i]).abs().max() / want[i].abs().max()
            assert err < 2e-5, f"cuts {cuts}, request {i}: {float(err):.3e}"
        assert bool((state[1] == 7.0).all()) and bool((prev[1] == 5.0).all()) and bool((prev[2] == 0).all())
        assert torch.equal(prev[3].cpu(), xs[0][-1]) and torch.equal(prev[0].cpu(), xs[1][-1])


@pytest.mark.parametrize("S, D, dt", [(1, 64, torch.float32), (2, 40, torch.bfloat16), (3, 1028, torch.float32), (4, 2048, torch.bfloat16), (5, 30, torch.float32),
                                      (7, 132, torch.float32), (8, 16, torch.bfloat16), (9, 24, torch.float32), (32, 7, torch.bfloat16), (4, 13000, torch.float32)])
def test_step_between_two_sublayers(S, D, dt):
    """A residual of S streams: what a sublayer reads before anything was added, the first add (from equal streams), later adds
    with a plain result, split-K slices, a bias, routed rows and two normed results, and the sum for picked rows."""
    from quench6k_b200 import ops
    g = torch.Generator().manual_seed(S * D)
    T, eps = 5, 1e-5
    rnd = lambda *s: torch.randn(*s, generator=g)
    tol = 2e-5 if dt == torch.float32 else 2e-2
    x, in_w, w = rnd(T, D), rnd(S), rnd(D)
    norm = lambda xs, iw: pg.rms_norm(sum(iw[s].double() * xs[s] for s in range(S)), w.double(), eps)
    close = lambda a, b, t=tol: float((a.double().cpu() - b).abs().max()) <= t * max(1.0, float(b.abs().max()))
    read = lambda iw: (iw.cuda(), w.cuda(), eps)
    xs = [x.double()] * S
    h = x.cuda()
    h, out = ops.hyper_step(h, S, None, read(in_w), None, dt)
    assert h.dim() == 2 and close(out, norm(xs, in_w))
    pair_row = torch.tensor([[1, 9], [0, 3], [7, 2], [4, 4], [5, 8]], dtype=torch.int32)
    for how in ("plain", "slices", "bias", "routed", "routed and plain", "pair", "pair with slices"):
        mix, out_w, in_w, bias = rnd(S, S) * (0.7 / S ** 0.5), rnd(S), rnd(S), rnd(D)
        a, b, wa, wb, py, pw = rnd(2, T, D), rnd(3, T, D), rnd(D), rnd(D), rnd(10, D), rnd(T, 2)
        add = {"mix": mix.cuda(), "out": out_w.cuda()}
        ad, bd = a.double(), b.double()
        routed = torch.stack([sum(pw[t, j].double() * py[pair_row[t, j]].double() for j in range(2)) for t in range(T)])
        if how == "plain":
            add["a"], y = a[0].contiguous().cuda(), ad[0]
        elif how == "slices":
            add["a"], y = a.cuda(), ad.sum(0)
        elif how == "bias":
            add.update(a=a[0].contiguous().cuda(), bias=bias.cuda())
            y = ad[0] + bias.double()
        elif how == "routed":
            add["weighted"], y = (py.cuda(), pair_row.cuda(), pw.cuda()), routed
        elif how == "routed and plain":
            add.update(a=a.cuda(), weighted=(py.cuda(), None, pw.cuda()))
            y = ad.sum(0) + torch.stack([sum(pw[t, j].double() * py[2 * t + j].double() for j in range(2)) for t in range(T)])
        else:
            many = how != "pair"
            add.update(a=a.cuda() if many else a[0].contiguous().cuda(), bias=bias.cuda(),
                       pair=((b if many else b[0]).contiguous().cuda(), wa.cuda(), wb.cuda(), 0.5, eps))
            left, right = (ad.sum(0) if many else ad[0]) + bias.double(), bd.sum(0) if many else bd[0]
            y = 0.5 * (pg.rms_norm(left, wa.double(), eps) + pg.rms_norm(right, wb.double(), eps))
            assert close(ops.normed_pair(add["a"], bias.cuda(), add["pair"][0], wa.cuda(), wb.cuda(), 0.5, eps), y, 2e-5)
        xs = [sum(mix[s, t].double() * xs[s] for s in range(S)) + out_w[t].double() * y for t in range(S)]
        # the sum over picked rows first (it stores nothing), then the step itself
        rows = torch.tensor([4, 1], dtype=torch.int32).cuda()
        same, total = ops.hyper_step(h, S, add, (torch.ones(S).cuda(), w.cuda(), eps), rows, dt)
        assert same is h and close(total, norm(xs, torch.ones(S))[[4, 1]]), how
        h, out = ops.hyper_step(h, S, add, read(in_w), None, dt)
        assert tuple(h.shape) == (T, S, D) and close(out, norm(xs, in_w)), how
        assert close(h, torch.stack(xs, 1), 2e-5), how
        xs = [h[:, s].double().cpu() for s in range(S)]


@pytest.mark.parametrize("hd, vd, slices", [(64, 64, 1), (128, 128, 3), (40, 40, 2), (24, 36, 1), (300, 20, 1)])
@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
def test_values_over_their_root_mean_square(hd, vd, slices, dt):
    """Both kernels that write the pages divide a head's value (biases included) by its root mean square."""
    from quench6k_b200 import ops
    g = torch.Generator().manual_seed(hd)
    T, Hq, Hkv, page = 6, 4, 2, 4
    N = Hq * hd + Hkv * hd + Hkv * vd
    qkv, bias = torch.randn(slices, T, N, generator=g), torch.randn(N, generator=g)
    ctx = helpers.make_context([T], [3], [[[2, 0, 1]]])
    pages = lambda n: torch.zeros(Hkv, 3, page, n, dtype=dt).cuda()
    total = qkv.double().sum(0) + bias.double()
    v = pg.rms_norm(total[:, (Hq + Hkv) * hd:].view(T, Hkv, vd), None, 1e-5)
    for name in ("qk_prep", "qkv_pages"):
        if name == "qk_prep" and vd != hd:
            continue
        kp, vp = pages(hd), pages(vd)
        x = (qkv if slices > 1 else qkv[0]).contiguous().cuda()
        if name == "qk_prep":
            ops.qk_prep(x, Hq, Hkv, hd, None, None, 1e-5, None, ctx.positions, ctx.req_of_token, ctx.block_tables[0], page, kp, vp, dt, bias=bias.cuda(), value_norm=True)
        else:
            ops.qkv_pages(x, Hq, Hkv, hd, vd, None, None, 1e-5, None, ctx.positions, ctx.req_of_token, ctx.block_tables[0], page, kp, vp, dt, bias=bias.cuda(),
                          value_norm=True)
        for t in range(T):
            p = 3 + t
            row = vp[:, [2, 0, 1][p // page], p % page].double().cpu()
            assert (row - v[t]).abs().max() < (1e-5 if dt == torch.float32 else 2e-2), name
            key = kp[:, [2, 0, 1][p // page], p % page].double().cpu()
            assert (key - total[t, Hq * hd:(Hq + Hkv) * hd].view(Hkv, hd)).abs().max() < (1e-4 if dt == torch.float32 else 5e-2), name


def test_small_kernels():
    """Gates per head (split-K slices), the norm of some columns, tanh of split-K slices, weights of the choice squared, and the
    output norm with a weight per head."""
    from quench6k_b200 import ops
    g = torch.Generator().manual_seed(9)
    rnd = lambda *s: torch.randn(*s, generator=g)
    for dt, tol in ((torch.float32, 1e-5), (torch.bfloat16, 3e-2)):
        for n in (20, 24, 136):
            a, p = rnd(5, 3 * n).to(dt), rnd(2, 5, 11)
            got = a.clone().cuda()
            ops.gate_heads(got, 3, p.cuda(), 7)
            want = a.double().view(5, 3, n) * torch.sigmoid(p.double().sum(0)[:, 7:10])[..., None]
            assert (got.double().cpu().view(5, 3, n) - want).abs().max() < tol
        for n, col in ((13, 5), (200, 5), (200, 8), (1500, 5), (1500, 8), (1024, 0), (4, 4)):
            x, w = rnd(4, n + 12), rnd(n)
            got = ops.norm_columns(x.cuda(), col, n, w.cuda(), 1e-5, dt).double().cpu()
            assert (got - pg.rms_norm(x.double()[:, col:col + n], w.double(), 1e-5)).abs().max() < 2 * tol, (n, col)
        z = rnd(3, 6, 10)
        assert (ops.activate(z.cuda(), 7, False, "tanh", dt).double().cpu() - torch.tanh(z.double().sum(0)[:, :7])).abs().max() < tol
        o, gate, w = rnd(5, 3 * 20), rnd(5, 60), rnd(3, 20)
        want = pg.rms_norm(o.double().view(5, 3, 20), w.double(), 1e-5).view(5, 60) * pg.silu(gate.double())
        assert (ops.delta_out(o.cuda(), gate.cuda(), 0, w.cuda(), 1e-5, 3, 20, dt).double().cpu() - want).abs().max() < 10 * tol
    z = rnd(40, 12)
    e1, w1 = ops.route_biased(z.cuda(), 3, None, 1.0, renorm=False)
    e2, w2 = ops.route_biased(z.cuda(), 3, None, 1.0, renorm=False, power=2)
    assert torch.equal(e1, e2) and torch.allclose(w2, w1 * w1) and torch.allclose(w1.cpu(), torch.sigmoid(z).gather(1, e1.cpu().long()))


# ------------------------------------------------------------------------------------------------- one mechanism alone
ONE = {
    "delta": (3, [gc.delta(4, 2, 16, 24, 4, 6, 10)]),
    "delta_one_key_head": (2, [gc.delta(3, 1, 40, 8, 2, 16, 5)]),
    "delta_one_tap": (1, [gc.delta(2, 2, 6, 10, 1, 4, 4)]),
    "delta_wide_keys": (4, [gc.delta(2, 1, 136, 20, 6, 8, 12)]),
    "delta_tensor_cores": (4, [gc.delta(4, 2, 64, 32, 4, 24, 16)]),
    "latent": (2, [gc.latent(3, 8, 12, 20, 24, 0.9)]),
    "latent_one_head": (5, [gc.latent(1, 24, 6, 7, 33, 0.6)]),
    "latent_borrowed": (3, [gc.latent(2, 12, 8, 10, 20, 0.8), gc.latent(4, 6, 10, 24, 20, 0.9, kv_from=0)]),
    "latent_tensor_cores": (3, [gc.latent(4, 32, 48, 64, 64, 0.15), gc.latent(2, 64, 32, 96, 64, 0.1, kv_from=0)]),
    "both": (3, [gc.both((4, 2, 16, 16, 0.7, 16, 300.0), (3, 16, 6))]),
    "both_no_rotation": (2, [gc.both((2, 1, 10, 14, 0.8, 0, 10.0), (2, 24, 9))]),
    "both_many_key_heads": (6, [gc.both((3, 3, 24, 8, 0.6, 10, 5000.0), (5, 6, 4))]),
    "both_tensor_cores": (4, [gc.both((4, 2, 64, 64, 0.35, 64, 10000.0), (2, 64, 16))]),
    "both_wide_heads": (4, [gc.both((2, 1, 112, 112, 0.3, 64, 10000.0), (1, 80, 16))]),
    "experts": (2, [gc.latent(1, 8, 8, 8, 8, 0.2, mlp=gc.moe(7, 3, 24))]),
    "all_experts": (3, [gc.latent(1, 8, 8, 8, 8, 0.2, mlp=gc.moe(3, 3, 16))]),
    "dense": (9, [gc.latent(1, 8, 8, 8, 8, 0.2, mlp=gc.ff(56))]),
}


@pytest.fixture(scope="module", params=sorted(ONE))
def single(request, tmp_path_factory):
    name = request.param
    streams, layers = ONE[name]
    wide = name.endswith("tensor_cores") or name == "both_wide_heads"
    folder = str(tmp_path_factory.mktemp(name))
    cfg, weights = gh.make_folder(folder, gc.few(layers, width=128 if wide else 48, page=16 if wide else 4, streams=streams), seed=3, init_std=0.3)
    reqs = {"long": helpers.random_tokens(230, cfg["vocab"], 1), "short": helpers.random_tokens(9, cfg["vocab"], 2),
            "one": helpers.random_tokens(1, cfg["vocab"], 3)}
    return name, folder, cfg, weights, reqs


@pytest.mark.parametrize("dtype", DTYPES)
def test_mechanism_alone_whole_prompt(single, dtype):
    name, folder, cfg, weights, reqs = single
    steps, mt = helpers.schedule_whole(reqs)
    gh.replay_and_compare(folder, cfg, weights, reqs, steps, mt, dtype, f"{name} whole")


@pytest.mark.parametrize("dtype", DTYPES)
def test_mechanism_alone_token_by_token(single, dtype):
    """Every token decoded alone from the first one on: each key is found through the cache, each state through its slot."""
    name, folder, cfg, weights, reqs = single
    steps, mt = helpers.schedule_tail(reqs, tail=10 ** 6)
    gh.replay_and_compare(folder, cfg, weights, reqs, steps, mt, dtype, f"{name} decoded")


@pytest.mark.parametrize("dtype", DTYPES)
def test_mechanism_alone_portions(single, dtype):
    name, folder, cfg, weights, reqs = single
    for seed in (0, 1):
        steps, mt = helpers.schedule_portions(reqs, seed=seed)
        gh.replay_and_compare(folder, cfg, weights, reqs, steps, mt, dtype, f"{name} portions")


def test_a_fault_would_show(single):
    """The premise of the tests above: a sink, a gate, a value norm or a convolution's reach left out, a key lost, a state that
    forgot its first tokens or a predecessor mistaken is far beyond the tolerance: the plain implementation, broken on
    purpose, differs from itself."""
    name, folder, cfg, weights, reqs = single
    toks = reqs["long"]
    a = gh.plain(cfg, weights, toks)
    far = lambda b, rows=slice(None): ((a[rows] - b).abs().max(-1).values / a.abs().max()) > 3 * gh.TOL["bfloat16"]
    changed = lambda **kw: gh.plain(cfg, {**weights, **{f"l0.mix.{n}": t for n, t in kw.pop("at").items()}}, toks)
    like = lambda n, v: torch.full_like(weights[f"l0.mix.{n}"], v)
    if name.startswith("both"):
        b = changed(at={"left.sink": like("left.sink", -80.0)})
        assert far(b).float().mean() > 0.1 or (a - b).abs().max() > 0.05 * a.abs().max(), "the sink left out does not show"
        assert far(changed(at={"left.g": like("left.g", 0.0)})).float().mean() > 0.15, "the heads' gates left out do not show"
        b = changed(at={"right.u": like("right.u", 0.0)})         # among the first tokens, while the state holds little
        assert far(b[:8], slice(0, 8)).float().mean() > 0.2, "the bonus left out does not show"
        assert far(changed(at={"right.mu.k": like("right.mu.k", 0.0)})).float().mean() > 0.15, "the token before does not show"
    if name.startswith("delta"):
        if cfg["layers"][0]["mixer"]["conv"] > 1:
            short = weights["l0.mix.k.conv"].clone()
            short[:, 0] = 0.0
            assert far(changed(at={"k.conv": short})).float().mean() > 0.15, "the convolution's first tap does not show"
        assert far(changed(at={"g2": like("g2", 0.0)})).float().mean() > 0.15, "the output gate left out does not show"
        assert far(changed(at={"a2": like("a2", 0.0)})).float().mean() > 0.05, "the decays' inputs left out do not show"
    if name.startswith(("delta", "both")):
        b = gh.plain(cfg, weights, toks[120:])
        moved = (a[120:] - b).abs().max(-1).values / a.abs().max()
        assert (moved[1:40] > gh.TOL["bfloat16"]).float().mean() > 0.5, "a lost state does not show in the next tokens"
        assert float(moved[100:].median()) > 100 * gh.TOL["float32"], "the state of the first 120 tokens no longer shows 100 tokens later"
    if name == "experts":
        others = {p: (e + 1) % cfg["layers"][0]["mlp"]["router"]["experts"] for p, e in gh.plain.chosen.items()}
        assert far(gh.plain(cfg, weights, toks, others)).float().mean() > 0.3, "another choice of experts does not show"


# ------------------------------------------------------------------------------------------------- a key that stands out
BEACON = 17


def _beacon(kind, push):
    """Channel 0 of the stream is the same positive number for every token and channel 1 is zero for all tokens but one.  The
    last entry of every key (outside the part that turns) reads channel 1 and the last entry of every query reads channel 0,
    in latent attention through the first entry of each low-rank vector: every query looks, above all, for that one token."""
    def doctor(w):
        gh.spread(w)
        w["embed"][:, 0], w["embed"][:, 1] = 1.0, 0.0
        w["embed"][BEACON, 1] = 4.0
        layers = sorted({n.split(".")[0] for n in w if n[0] == "l" and n[1].isdigit()})
        for L in layers:
            w[f"{L}.norm1"].fill_(1.0)
            w[f"{L}.mix.left.o" if kind == "left" else f"{L}.mix.o"][:2] = 0.0            # the sublayer's result leaves both channels alone
            if kind == "left":
                w[f"{L}.mix.left.o.b"][:2] = 0.0
                w[f"{L}.mix.right.o"][:2] = 0.0
        for L in layers:
            if kind == "left":
                G, H, dim = 1, 2, 8
                for n, heads, channel, size in (("k", G, 1, 10.0), ("q", H, 0, push)):
                    m, b = w[f"{L}.mix.left.{n}"].view(heads, dim, -1), w[f"{L}.mix.left.{n}.b"].view(heads, dim)
                    m[:, dim - 1], b[:, dim - 1] = 0.0, 0.0
                    m[:, dim - 1, channel] = size
                w[f"{L}.mix.left.g"].zero_()
                w[f"{L}.mix.left.out"].fill_(2.0)
            else:
                if f"{L}.mix.dkv" in w:
                    w[f"{L}.mix.dkv"][0] = 0.0
                    w[f"{L}.mix.dkv"][0, 1] = 6.0
                    w[f"{L}.mix.dkv.norm"][0] = 1.0
                w[f"{L}.mix.dq"][0] = 0.0
                w[f"{L}.mix.dq"][0, 0] = 3.0
                w[f"{L}.mix.dq.norm"][0] = 1.0
                H = 2
                for n, size in (("uk", 8.0), ("uq", push)):
                    m = w[f"{L}.mix.{n}"].view(H, 8, -1)
                    m[:, 7] = 0.0
                    m[:, 7, 0] = size
                w[f"{L}.mix.o"].mul_(3.0)
    return doctor


FAR = {"left": [gc.both((2, 1, 8, 8, 1.0, 4, 100.0), (1, 8, 4))],
       "latent": [gc.latent(2, 8, 8, 6, 12, 1.0)],
       "borrowed": [gc.latent(2, 8, 8, 6, 12, 1.0), gc.latent(2, 8, 5, 9, 12, 1.0, kv_from=0)]}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", sorted(FAR))
def test_a_key_far_away_and_at_page_borders(tmp_path, which, dtype):
    """The token every query looks for stands at the start, on both sides of a page border and inside a page of unequal requests,
    and positions hundreds of tokens on (in the prompt, in portions and decoded one by one) still rest on it."""
    cfg, weights = gh.make_folder(str(tmp_path), gc.few(FAR[which], page=8, streams=2), seed=12, init_std=0.15, doctor=_beacon("left" if which == "left" else "latent", 4.0))
    reqs = {}
    for i, place in enumerate((0, 7, 8, 43, 200)):
        toks = [t if t != BEACON else 3 for t in helpers.random_tokens(330 + i, cfg["vocab"], 6 + i)]
        toks[place] = BEACON
        reqs[f"at{place}"] = toks
        without = list(toks)
        without[place] = 3
        want, other = gh.plain(cfg, weights, toks), gh.plain(cfg, weights, without)
        assert float((want[290:] - other[290:]).abs().max(-1).values.min()) > 0.05 * float(want.abs().max()), f"positions far from {place} do not rest on the token"
    for what, (steps, mt) in {"whole": helpers.schedule_whole(reqs), "decoded": helpers.schedule_tail(reqs, tail=60),
                              "portions": helpers.schedule_portions(reqs, seed=4), "mixed": helpers.schedule_mixed(reqs, 8, seed=2, max_live=3)}.items():
        gh.replay_and_compare(str(tmp_path), cfg, weights, reqs, steps, mt, dtype, f"far key, {which}, {what}")


# ------------------------------------------------------------------------------------------------- whole models
LENGTHS = {"G1": [71, 130, 45, 96, 64, 33, 1, 58, 77], "G2": [85, 140, 37, 101, 2, 50, 90, 125, 44], "G3": [90, 217, 129, 48, 75, 40, 150, 66, 83],
           "G4": [70, 33, 131, 20, 64, 3, 95, 41, 58]}


@pytest.fixture(scope="module", params=sorted(LENGTHS))
def model(request, tmp_path_factory):
    name = request.param
    folder = str(tmp_path_factory.mktemp(name))
    cfg, weights = gh.make_folder(folder, gc.get(name), seed=7, init_std=0.1)
    reqs = {f"r{i}": helpers.random_tokens(n, cfg["vocab"], 100 + i) for i, n in enumerate(LENGTHS[name])}
    return {"name": name, "folder": folder, "cfg": cfg, "weights": weights, "requests": reqs}


@pytest.mark.parametrize("dtype", DTYPES)
def test_model_whole(model, dtype):
    steps, mt = helpers.schedule_whole(model["requests"])
    gh.replay_and_compare(model["folder"], model["cfg"], model["weights"], model["requests"], steps, mt, dtype, model["name"] + " whole")


def test_the_streams_after_every_layer(model):
    """The sum of the streams after each layer against the plain implementation's, float32: a layer that is wrong is named."""
    from quench6k_b200.engine import ModelRunner
    toks = model["requests"]["r0"]
    want = []
    pg.forward(model["cfg"], model["weights"], toks, layers_out=want)
    runner = ModelRunner.from_folder(model["folder"], dtype="float32", page_size=model["cfg"]["kv_page_size"], num_pages=64, max_requests=2)
    got = gh.streams_of(runner, toks)
    assert len(got) == len(want)
    for i, (a, b) in enumerate(zip(got, want)):
        err = float((a.double().cpu() - b).abs().max() / b.abs().max())
        assert err < 1e-4, f"{model['name']}: the streams after layer {i} ({model['cfg']['layers'][i]['type']}): {err:.3e}"


@pytest.mark.parametrize("dtype", DTYPES)
def test_model_prefill_then_decode(model, dtype):
    steps, mt = helpers.schedule_tail(model["requests"], tail=40)
    gh.replay_and_compare(model["folder"], model["cfg"], model["weights"], model["requests"], steps, mt, dtype, model["name"] + " tail")


@pytest.mark.parametrize("dtype", DTYPES)
def test_model_portions(model, dtype):
    steps, mt = helpers.schedule_portions(model["requests"], seed=5)
    gh.replay_and_compare(model["folder"], model["cfg"], model["weights"], model["requests"], steps, mt, dtype, model["name"] + " portions")


@pytest.mark.parametrize("dtype", DTYPES)
def test_model_mixed_batches_reuse_pages_and_slots(model, dtype):
    """Up to four live requests, unequal portions beside single tokens, requests that sit steps out; nine requests go
    through four slots and a pool of the live requests' size, so every slot and most pages are used again."""
    page = model["cfg"]["kv_page_size"]
    for seed in (0, 1):
        steps, mt = helpers.schedule_mixed(model["requests"], page, seed=seed, max_live=4)
        got = gh.replay_and_compare(model["folder"], model["cfg"], model["weights"], model["requests"], steps, mt, dtype,
                                    model["name"] + " mixed", max_requests=4)
    if dtype == "float32":
        # and the same requests each alone: what else is in the batch, and which pages and slots are used, changes nothing
        steps, mt = helpers.schedule_whole(model["requests"])
        outputs, _ = helpers.run_replay(model["folder"], dtype, steps, mt)
        alone = helpers.collect(model["requests"], steps, outputs)
        for rid in model["requests"]:
            gh.assert_close(got[rid], alone[rid], dtype, f"{model['name']} {dtype} {rid} batched against alone", tol=2e-5)


@pytest.mark.parametrize("dtype", DTYPES)
def test_model_many_decoding_together(model, dtype):
    page = model["cfg"]["kv_page_size"]
    reqs = {rid: t for rid, t in model["requests"].items() if len(t) > 12}
    steps, mt = helpers.schedule_wide_decode(reqs, page)
    gh.replay_and_compare(model["folder"], model["cfg"], model["weights"], reqs, steps, mt, dtype, model["name"] + " wide decode",
                          max_requests=len(reqs))


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(model, dtype):
    """A short prompt and hundreds of tokens decoded one by one: pages pass over decoded tokens, the recurrent states run long,
    the decode steps are replayed from a recorded graph."""
    reqs = {"d": helpers.random_tokens(320, model["cfg"]["vocab"], 9)}
    steps, mt = helpers.schedule_tail(reqs, tail=310)
    gh.replay_and_compare(model["folder"], model["cfg"], model["weights"], reqs, steps, mt, dtype, model["name"] + " long decode")


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_long_prompt(model, dtype):
    """A prompt of 1,100 tokens whole, in portions, and with its last tokens decoded: recurrent states a thousand tokens old."""
    if model["name"] not in ("G1", "G3"):
        pytest.skip("two of the models are enough for the length")
    reqs = {"p": helpers.random_tokens(1100, model["cfg"]["vocab"], 21)}
    for what, (steps, mt) in {"whole": helpers.schedule_whole(reqs), "portions": helpers.schedule_portions(reqs, seed=8),
                              "tail": helpers.schedule_tail(reqs, tail=40)}.items():
        gh.replay_and_compare(model["folder"], model["cfg"], model["weights"], reqs, steps, mt, dtype, f"{model['name']} long prompt {what}")


def test_greedy_generation_through_the_engine(model):
    """Engine.generate (scheduler, continuous batching, device-side argmax, tokens that stay on the device for the next step,
    CUDA graphs) against greedy decoding with the plain implementation, float32; prompts of unequal length in one engine
    with few pages."""
    import quench6k_b200 as q
    cfg, weights = model["cfg"], model["weights"]
    prompts = [helpers.random_tokens(n, cfg["vocab"], 50 + n) for n in (5, 23, 1, 40, 12, 31)]
    page = cfg["kv_page_size"]
    eng = q.Engine.from_folder(model["folder"], dtype="float32", page_size=page, num_pages=4 * (64 // page + 2), max_requests=4,
                               max_batch_tokens=32)
    outs = eng.generate(prompts, q.SamplingParams(max_tokens=12, temperature=0))
    for prompt, out in zip(prompts, outs):
        toks = list(prompt)
        for i in range(12):
            logits = gh.plain(cfg, weights, toks)[-1]
            top2 = logits.topk(2).values
            if float(top2[0] - top2[1]) < 1e-3 * float(logits.abs().max()):
                break                                  # a near-tie: float32 may pick either; the continuation is not comparable
            assert out.tokens[i] == int(logits.argmax()), f"{model['name']}: prompt of {len(prompt)}, generated token {i}"
            toks.append(out.tokens[i])
    eng.runner.manager.check()


def test_command_line_generates(model):
    """`generate` of the command line on a Gunenex model folder: the model class comes from config.json."""
    if model["name"] != "G1":
        pytest.skip("one model is enough for the command line")
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
        logits = gh.plain(cfg, weights, toks)[-1]
        top2 = logits.topk(2).values
        if float(top2[0] - top2[1]) < 1e-3 * float(logits.abs().max()):
            return
        toks.append(int(logits.argmax()))
    assert "prompt: 11 tokens" in r.stdout and f"ids: {toks[11:]}" in r.stdout
