"""The kernels and options that came with the Soporax decoder, each alone against float64 torch arithmetic, at sizes of no
model."""
import math

import pytest
import torch

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
TYPES = [torch.float32, torch.bfloat16]


def K():
    from exl3_server_b200.ops import kernels
    return kernels


def close(got, want, dt, what=""):
    got, want = got.double().cpu(), want.double().cpu()
    err = float((got - want).abs().max()) / max(1e-30, float(want.abs().max()))
    assert err <= (2e-5 if dt == torch.float32 else 2e-2), (what, err)


@pytest.mark.parametrize("dt", TYPES)
@pytest.mark.parametrize("H", [96, 101, 7, 1028, 2304, 8192, 8200])
@pytest.mark.parametrize("top", [0, 1, 3, 9])
def test_residual_step(dt, H, top):
    """Widths of every form (one to eight pieces a thread, odd ones, rows longer than registers); both outputs, one of them
    or none; picks; the embedding's row by id or in place; a vector; with and without the norm."""
    g = torch.Generator().manual_seed(H + top)
    k_ = K()
    T, V = 5, 11
    h0 = torch.randn(T, H, generator=g)
    a, b = torch.randn(T, H, generator=g).to(dt), torch.randn(T, H, generator=g)
    y = torch.randn(T * max(1, top), H, generator=g)
    ids = torch.tensor([3, 10, 0, 3, 7], dtype=torch.int32)
    table, rows = torch.randn(V, H, generator=g).to(dt), torch.randn(T, H, generator=g)
    vec = torch.randn(H, generator=g)
    w = (1 + 0.3 * torch.randn(H, generator=g)).to(dt)
    d = lambda t: t.to(DEV) if t is not None else None
    for use_a, use_b, emb, use_vec, norm in ((1, 1, "ids", 1, 1), (1, 0, None, 1, 1), (0, 0, "rows", 0, 1), (1, 0, "ids", 0, 0),
                                             (0, 1, None, 0, 1), (0, 0, None, 1, 0)):
        h = h0.clone().to(DEV)
        entry = None
        if emb or use_vec:
            e = {"ids": table, "rows": rows, None: None}[emb]
            entry = (d(e), d(ids) if emb == "ids" else None, 1.5, d(vec) if use_vec else None)
        x = k_.residual_step(h, d(a) if use_a else None, d(b) if use_b else None, (d(y), top, 0.3) if top else None, 0.7, entry,
                             (d(w), 1e-5, dt) if norm else None)
        want = torch.zeros(T, H, dtype=torch.float64)
        if use_a:
            want = want + a.double()
        if use_b:
            want = want + b.double()
        if top:
            want = want + 0.3 * y.double().reshape(T, top, H).sum(1)
        want = h0.double() + 0.7 * want
        if emb:
            want = want + 1.5 * (table[ids.long()].double() if emb == "ids" else rows.double())
        if use_vec:
            want = want + vec.double()
        close(h, want, torch.float32, (use_a, use_b, emb, use_vec))
        if norm:
            close(x, want / torch.sqrt((want * want).mean(-1, keepdim=True) + 1e-5) * w.double(), dt, "norm")
        else:
            assert x is None
        # a token alone: the same bits
        h1 = h0[2:3].clone().to(DEV)
        if emb == "rows":
            entry = (d(rows[2:3]), None, 1.5, entry[3])
        elif emb:
            entry = (entry[0], d(ids[2:3]), 1.5, entry[3])
        k_.residual_step(h1, d(a[2:3]) if use_a else None, d(b[2:3]) if use_b else None,
                         (d(y[2 * top:3 * top]), top, 0.3) if top else None, 0.7, entry, None)
        assert torch.equal(h1[0], h[2])


def test_plans_from_tables_in_one_launch():
    """Layers with different numbers of experts, picks and tile sizes; more layers than one launch takes."""
    g = torch.Generator().manual_seed(5)
    k_ = K()
    V, T = 40, 77
    ids = torch.randint(0, V, (T,), generator=g, dtype=torch.int32)
    shapes = [(6, 2, 4), (1, 1, 32), (130, 9, 128), (5, 5, 4), (17, 1, 32)] * 11
    layers = []
    for E, top, rows in shapes:
        table = torch.rand(V, E, generator=g).argsort(dim=1)[:, :top].to(torch.int32).contiguous()
        layers.append((table.to(DEV), E, rows))
    plans = k_.moe_table_plans(ids.to(DEV), layers)
    assert len(plans) == len(layers)
    for (table, E, rows), (E_, top, _), (order, plan) in zip(layers, shapes, plans):
        order, plan, table = order.cpu(), plan.cpu(), table.cpu()
        assert int(plan[1]) == T * top and sorted(order.tolist()) == list(range(T * top))
        seen = 0
        for i in range(int(plan[0])):
            e, first, n = plan[4 + 3 * i:7 + 3 * i].tolist()
            assert first == seen and 1 <= n <= rows
            for p in order[first:first + n].tolist():
                assert int(table[int(ids[p // top]), p % top]) == e
            seen += n
        assert seen == T * top


@pytest.mark.parametrize("act", ["silu", "gelu"])
def test_gated_experts_in_the_products_epilogues(act):
    """Gate and up rows in turn, act(gate) * up out of all three products, at widths that fill no tile; pairs in one tile and
    in many."""
    g = torch.Generator().manual_seed(9)
    k_ = K()
    f = {"silu": torch.nn.functional.silu, "gelu": torch.nn.functional.gelu}[act]
    for kind, T, dt, W, inner in (("tile", 20, torch.float32, 41, 13), ("tile", 70, torch.bfloat16, 96, 33), ("few", 1, torch.bfloat16, 96, 40),
                                  ("few", 9, torch.bfloat16, 1032, 27), ("tc", 400, torch.bfloat16, 96, 72), ("tc", 300, torch.bfloat16, 136, 200)):
        top, E = 2, 5
        x = torch.randn(T, W, generator=g).to(dt)
        idx = torch.randint(0, E, (T, top), generator=g, dtype=torch.int32)
        wg, wu = ((torch.randn(E, inner, W, generator=g) / math.sqrt(W)).to(dt) for _ in range(2))
        w = torch.stack([wg, wu], dim=2).reshape(E, 2 * inner, W).contiguous()
        want = []
        for p in range(T * top):
            e, xr = int(idx[p // top, p % top]), x[p // top].double()
            want.append(f(wg[e].double() @ xr) * (wu[e].double() @ xr))
        want = torch.stack(want)
        order, plan = k_.moe_plan(idx.to(DEV), E, k_.moe_tile_rows(kind))
        if kind == "tc":
            mid = k_.moe_gemm_tc(k_.moe_gather(x.to(DEV), top, order, plan), w.to(DEV), order, plan, dt, act=act, glu=True)
            want_rows = want[order.long().cpu()]
            close(mid, want_rows, dt, (kind, T))
            own = k_.moe_gemm_tc(k_.moe_gather(x.to(DEV), top, order, plan), w.to(DEV), order, plan, torch.float32, act=act, glu=True)
            close(own, want, dt, (kind, T, "float32 at the pairs' places"))
        else:
            for out_dt in ([dt] if kind == "tile" else [dt, torch.float32]):
                mid = (k_.moe_gemm if kind == "tile" else k_.moe_gemv)(x.to(DEV), top, w.to(DEV), order, plan, out_dt, act=act, glu=True)
                assert mid.shape == (T * top, inner)
                close(mid, want, dt, (kind, T))
    assert k_.moe_tc_status() == 0


@pytest.mark.parametrize("y_dt, g_dt", [(torch.float32, torch.float32), (torch.bfloat16, torch.bfloat16), (torch.bfloat16, torch.float32)])
@pytest.mark.parametrize("T, n, off, ld", [(1, 8, 0, 8), (7, 40, 16, 72), (130, 33, 5, 51), (3, 2048, 8, 2064)])
def test_sigmoid_factors_in_place(y_dt, g_dt, T, n, off, ld):
    g = torch.Generator().manual_seed(T + n)
    y, a = torch.randn(T, n, generator=g).to(y_dt), (4.0 * torch.randn(T, ld, generator=g)).to(g_dt)
    got = K().sigmoid_mul(y.to(DEV), a.to(DEV)[:, off:off + n])
    close(got, y.double() * torch.sigmoid(a[:, off:off + n].double()), y_dt)


def rotated(x, pos, f, layout, mscale, rot):
    """x [T, n] with its first ``rot`` features rotated."""
    y = x.clone()
    half = rot // 2
    for i in range(half):
        a = pos.double() * f[i]
        u, v = (2 * i, 2 * i + 1) if layout else (i, i + half)
        y[:, u] = (x[:, u] * a.cos() - x[:, v] * a.sin()) * mscale
        y[:, v] = (x[:, v] * a.cos() + x[:, u] * a.sin()) * mscale
    return y


@pytest.mark.parametrize("dt", TYPES)
@pytest.mark.parametrize("layout, mscale", [(0, 1.0), (1, 1.0), (1, 1.31), (0, 0.9)])
@pytest.mark.parametrize("H, qr, r, rd, rot", [(3, 20, 24, 8, 8), (0, 130, 200, 64, 64), (0, 16, 33, 10, 6)])
def test_latent_rows_with_both_layouts(dt, layout, mscale, H, qr, r, rd, rot):
    """The step between the joint projection and the rest: both layouts of the rotation, a factor on sines and cosines, with
    gates per head and without gates."""
    g = torch.Generator().manual_seed(qr + r)
    k_ = K()
    up = lambda n: (n + 15) // 16 * 16
    row, rank_pad = up(up(r) + rd), up(r)
    tok_seq = torch.tensor([0] * 5 + [1] * 2, dtype=torch.int32)
    tok_pos = torch.tensor([62, 63, 64, 65, 66, 0, 1], dtype=torch.int32)
    T = 7
    a = torch.randn(T, qr + r + rd + H + 5, generator=g).to(dt)
    wq, wkv = 1 + 0.3 * torch.randn(qr, generator=g), 1 + 0.3 * torch.randn(r, generator=g)
    f = torch.tensor([100.0 ** (-2.0 * i / max(1, rot)) for i in range(rot // 2)], dtype=torch.float64)
    bt = torch.tensor([[3, 1], [0, -1]], dtype=torch.int32)
    pool = torch.full((5, 1, 64, row), 7.0, dtype=dt, device=DEV)
    cq, gate = k_.latent_prep(a.to(DEV), 0, qr, wq.to(DEV), qr, r, rd, wkv.to(DEV), qr + r + rd, H, 1e-5, k_.rotary_table(f).to(DEV),
                              rot, tok_pos.to(DEV), tok_seq.to(DEV), bt.to(DEV), 64, pool, row, rank_pad, dt, layout=layout, mscale=mscale)
    ad = a.double()
    nrm = lambda x, w: x / torch.sqrt((x * x).mean(-1, keepdim=True) + 1e-5) * w.double()
    close(cq, nrm(ad[:, :qr], wq), dt, "query latent")
    if H:
        close(gate, torch.sigmoid(ad[:, qr + r + rd:qr + r + rd + H]), torch.float32, "gates")
    else:
        assert gate is None
    want = torch.full(pool.shape, 7.0, dtype=torch.float64)
    c, kr = nrm(ad[:, qr:qr + r], wkv), rotated(ad[:, qr + r:qr + r + rd], tok_pos, f, layout, mscale, rot)
    for t in range(T):
        pg, at = int(bt[int(tok_seq[t]), int(tok_pos[t]) // 64]), int(tok_pos[t]) % 64
        want[pg, 0, at] = 0
        want[pg, 0, at, :r] = c[t]
        want[pg, 0, at, rank_pad:rank_pad + rd] = kr[t]
    close(pool, want, dt, "rows")


@pytest.mark.parametrize("dt", TYPES)
@pytest.mark.parametrize("layout, mscale", [(0, 1.0), (1, 1.2)])
@pytest.mark.parametrize("T, H, Kf, N, rd, rot", [(1, 3, 24, 40, 8, 8), (9, 16, 128, 256, 32, 32), (70, 2, 10, 36, 6, 4), (5, 4, 520, 48, 0, 0)])
def test_products_per_head_with_gates_per_feature(dt, layout, mscale, T, H, Kf, N, rd, rot):
    g = torch.Generator().manual_seed(T + N)
    k_ = K()
    tail, head = (N + 15) // 16 * 16, ((N + 15) // 16 * 16 + rd + 15) // 16 * 16
    x = torch.randn(T, H * (Kf + rd), generator=g).to(dt)
    w = (torch.randn(H, Kf, N, generator=g) / math.sqrt(Kf)).to(dt)
    gates = (3.0 * torch.randn(T, H * N + 24, generator=g)).to(dt)
    pos = torch.randint(0, 5000, (T,), generator=g, dtype=torch.int32)
    f = torch.tensor([1000.0 ** (-2.0 * i / max(1, rot)) for i in range(rot // 2)], dtype=torch.float64)
    out = torch.full((T, H * head), 5.0, dtype=dt, device=DEV)
    k_.head_gemm(x.to(DEV), H * (Kf + rd), Kf + rd, w.to(DEV), out, H * head, head, T, H, Kf, N, rot_dim=rd, rot=rot,
                 inv_freq=k_.rotary_table(f).to(DEV) if rot else None, tok_pos=pos.to(DEV), tail_off=tail, layout=layout,
                 mscale=mscale, gate=gates.to(DEV)[:, 8:8 + H * N])
    xd = x.double().reshape(T, H, Kf + rd)
    want = torch.zeros(T, H, head, dtype=torch.float64)
    want[:, :, :N] = torch.einsum("thk,hkn->thn", xd[:, :, :Kf], w.double()) * torch.sigmoid(gates[:, 8:8 + H * N].double()).reshape(T, H, N)
    for h in range(H):
        if rd:
            want[:, h, tail:tail + rd] = rotated(xd[:, h, Kf:], pos, f, layout, mscale, rot)
    close(out.reshape(T, H, head), want, dt)


@pytest.mark.parametrize("dt", TYPES)
@pytest.mark.parametrize("H, G, d, dv, off, gap", [(4, 2, 24, 16, 8, 3), (40, 8, 64, 64, 8, 0), (3, 1, 10, 6, 5, 1), (300, 1, 8, 8, 0, 4)])
def test_gates_beside_queries_and_keys(dt, H, G, d, dv, off, gap):
    """Both forms of the step before the attention leave the heads' gates as float32 factors; more heads than threads."""
    g = torch.Generator().manual_seed(H)
    k_ = K()
    T, n_pages = 3, 4
    dp, dvp = (d + 7) // 8 * 8, (dv + 7) // 8 * 8
    g_off = off + (H + G) * d + G * dv + gap
    ld = (g_off + H + 7) // 8 * 8
    x = (2.0 * torch.randn(T, ld, generator=g)).to(dt)
    kp, vp = (torch.zeros(n_pages, G, 64, n, dtype=dt, device=DEV) for n in (dp, dvp))
    args = (H, G, d, dv, dp, dvp, 1, None, None, 1e-5, 0, 0, None, 1.0, 1.0, None, torch.tensor([5, 6, 0], dtype=torch.int32, device=DEV),
            torch.tensor([0, 0, 1], dtype=torch.int32, device=DEV), torch.tensor([[2], [1]], dtype=torch.int32, device=DEV), 64, dt)
    q, _, gate = k_.qk_prep(x.to(DEV), off, off + H * d, off + (H + G) * d, *args, kp, vp, gate_off=g_off)
    close(gate, torch.sigmoid(x[:, g_off:g_off + H].double()), torch.float32)
    q2, _ = k_.qk_prep(x.to(DEV), off, off + H * d, off + (H + G) * d, *args, kp, vp)
    assert torch.equal(q, q2)


class Case:
    """Sequences over shuffled pages, queries of one token each, a window, a sink per head and a factor per head."""

    def __init__(self, H, G, d, dv, window, dt, queries, lens=(700, 1, 130, 65), seed=4):
        g = torch.Generator().manual_seed(seed)
        n_pages, width = 40, 12
        perm = torch.randperm(n_pages, generator=g)
        bt = torch.full((len(lens), width), -1, dtype=torch.int32)
        at = 0
        for b, n in enumerate(lens):
            need = (n + 63) // 64
            bt[b, :need] = perm[at:at + need].int()
            at += need
        kp, vp = torch.randn(n_pages, G, 64, d, generator=g).to(dt), torch.randn(n_pages, G, 64, dv, generator=g).to(dt)
        self.T = len(queries)
        q = torch.randn(self.T, H * d, generator=g).to(dt)
        sink, gate = 3.0 * torch.rand(H, generator=g) - 1.0, torch.rand(self.T, H, generator=g)
        self.scale = 0.9 / math.sqrt(d)
        want = torch.zeros(self.T, H, dv, dtype=torch.float64)
        for t, (b, p) in enumerate(queries):
            js = torch.arange(max(0, p - window + 1) if window else 0, p + 1)
            pg = bt[b, js // 64].long()
            kk, vv = kp[pg, :, js % 64].double(), vp[pg, :, js % 64].double()
            for h in range(H):
                s = kk[:, h // (H // G)] @ q[t, h * d:(h + 1) * d].double() * self.scale
                m = float(s.max())
                e = torch.exp(s - m)
                want[t, h] = float(gate[t, h]) * (e / (e.sum() + math.exp(float(sink[h]) - m))) @ vv[:, h // (H // G)]
        self.want = want
        if window:                                     # pages that no query of a sequence sees are given back
            for b in range(len(lens)):
                first = min([max(0, p - window + 1) // 64 for s, p in queries if s == b], default=0)
                bt[b, :first] = -1
        self.q, self.kp, self.vp, self.bt = q.to(DEV), kp.to(DEV), vp.to(DEV), bt.to(DEV)
        self.tok_seq = torch.tensor([b for b, _ in queries], dtype=torch.int32, device=DEV)
        self.tok_pos = torch.tensor([p for _, p in queries], dtype=torch.int32, device=DEV)
        self.sink, self.gate = sink.to(DEV), gate.to(DEV)


@pytest.mark.parametrize("dt", TYPES)
@pytest.mark.parametrize("H, G, d, dv, window", [(4, 2, 24, 16, 50), (6, 2, 16, 40, 1), (2, 1, 64, 64, 0), (20, 1, 16, 16, 129),
                                                 (5, 5, 160, 136, 300)])
def test_gated_heads_on_the_cuda_cores(dt, H, G, d, dv, window):
    c = Case(H, G, d, dv, window, dt, [(0, 699), (0, 450), (0, 256), (0, 255), (0, 0), (1, 0), (2, 129), (2, 127), (3, 64), (3, 63)])
    k_ = K()
    for split in (1024, 256, 64):
        n = (700 + split - 1) // split
        for T in (c.T, 2):                             # two tokens: the merge inside the attention kernel
            scratch = torch.zeros(k_.attn_tokens_scratch_bytes(T, H, dv, n) // 4 + 1, device=DEV)
            out = torch.empty(T, H * dv, dtype=dt, device=DEV)
            k_.attn_tokens_ex(c.q[:T], H * d, out, c.kp, c.vp, c.bt, c.tok_pos[:T], c.tok_seq[:T], T, H, G, d, dv, 64, window, 0,
                              True, c.scale, split, n, scratch, sink_vals=c.sink, gate=c.gate[:T].contiguous())
            close(out.reshape(T, H, dv), c.want[:T], dt, f"split {split}, {T} tokens")


@pytest.mark.parametrize("H, G, d, window", [(4, 2, 64, 50), (8, 1, 128, 300), (12, 1, 64, 1), (4, 4, 128, 65), (32, 2, 64, 128), (6, 2, 64, 0)])
def test_gates_windows_and_sinks_for_single_tokens(H, G, d, window):
    """The decode kernel's ways of ending a row (one chunk; chunks merged through scratch; inside a block or a cluster), with
    groups of heads split and in twins, under windows that begin anywhere in a page and in a chunk."""
    queries = [(0, 699), (1, 0), (2, 129), (3, 64), (0, 448), (0, 447), (0, 511), (0, 576), (2, 64)]
    c = Case(H, G, d, d, window, torch.bfloat16, queries)
    k_ = K()
    group = H // G
    for split, in_block, head_split, twins in ((1024, 0, 1, 1), (256, 0, 1, 1), (64, 0, 2, 1), (256, 1, 1, 1), (128, 2, 1, 1),
                                               (256, 1, 2, 2), (128, 2, 2, 2)):
        if group % head_split or (twins == 2 and group // head_split > 8):
            continue
        n = (700 + split - 1) // split
        scratch = torch.zeros(k_.attn_tokens_scratch_bytes(c.T, H, d, n) // 4 + 1, device=DEV) if n > 1 and not in_block else None
        out = torch.empty(c.T, H * d, dtype=torch.bfloat16, device=DEV)
        k_.attn_decode(c.q, H * d, out, c.kp, c.vp, c.bt, c.tok_pos, c.tok_seq, c.T, H, G, d, 64, window, c.scale, split, n, scratch,
                       in_block=in_block, head_split=head_split, twins=twins, sink=True, sink_vals=c.sink, gate=c.gate)
        close(out.reshape(c.T, H, d), c.want, torch.bfloat16, f"split {split} in_block {in_block} heads / {head_split}")
    assert k_.attn_decode_status() == 0


@pytest.mark.parametrize("nh, nkv, hd", [(4, 2, 64), (8, 1, 64), (4, 2, 128), (5, 1, 128)])
@pytest.mark.parametrize("window", [0, 100, 1])
def test_gated_heads_for_prompts(nh, nkv, hd, window):
    """Whole prompts, portions after earlier context and single rows through the tcgen05 kernel in each of its forms, with a
    factor per token and head."""
    from test_kernels_gpu import PagedCase
    k_ = K()
    case = PagedCase(lens=[300, 64, 1, 700, 65, 128, 129], new=[300, 64, 1, 200, 65, 1, 129], nh=nh, nkv=nkv, hd=hd,
                     dtype=torch.bfloat16, seed=hd + nh + window)
    T = case.q.shape[0]
    buf = case.q.reshape(T, nh * hd).to(DEV).contiguous()
    scale = 1.3 / math.sqrt(hd)
    g = torch.Generator().manual_seed(3)
    sink, gate = 3.0 * torch.rand(nh, generator=g) - 1.0, torch.rand(T, nh, generator=g)
    outs, t, G = [], 0, nh // nkv
    for b, (n, m) in enumerate(zip(case.lens, case.new)):
        k, v = (a[b].double().repeat_interleave(G, dim=1) for a in (case.k, case.v))
        s = torch.einsum("qhd,khd->hqk", case.q[t:t + m].double(), k) * scale
        back = torch.arange(n - m, n)[:, None] - torch.arange(n)[None, :]
        s = s.masked_fill((back < 0) | ((back >= window) if window else (back < 0)), float("-inf"))
        mx = s.max(dim=-1, keepdim=True).values
        e = torch.exp(s - mx)
        o = torch.einsum("hqk,khd->qhd", e / (e.sum(-1, keepdim=True) + torch.exp(sink.double()[:, None, None] - mx)), v)
        outs.append(o * gate[t:t + m].double()[:, :, None])
        t += m
    want = torch.cat(outs).reshape(-1, nh * hd)
    tile_seq, tile_q0 = case.tiles(128)
    got = []
    for variant in ((0, 1, 2, 3) if hd == 64 else (0, 1, 3)):
        o = torch.full((T, nh * hd), 3.0, device=DEV, dtype=torch.bfloat16)
        k_.attn_prefill_tc(buf, buf.stride(0), o, case.k_pool, case.v_pool, case.table, case.row_start, case.row_pos0,
                           tile_seq, tile_q0, tile_seq.numel(), nh, nkv, hd, 64, window, scale, variant=variant, sink=True,
                           sink_vals=sink.to(DEV), gate=gate.to(DEV))
        err = float((o.double().cpu() - want).abs().max()) / float(want.abs().max())
        assert err <= 1e-2, (variant, err)
        got.append(o)
    for o in got[1:]:
        assert torch.equal(got[0], o)
    assert k_.attn_prefill_tc_status() == 0
