"""The kernels and options that came with the Tunavik decoder, each alone against float64 torch arithmetic, at sizes of no
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
@pytest.mark.parametrize("H, norm", [(96, True), (101, True), (7, False), (4500, True)])
def test_embedding_with_sinusoids(dt, H, norm):
    """Odd widths, rows longer than a thread keeps in registers, positions far out."""
    g = torch.Generator().manual_seed(H)
    k_ = K()
    V = 31
    pos = torch.tensor([0, 1, 2, 63, 64, 1000, 4095, 70000, 300000], dtype=torch.int32)
    ids = torch.randint(0, V, (len(pos),), generator=g, dtype=torch.int32)
    table = torch.randn(V, H, generator=g).to(dt)
    w = 1.0 + 0.3 * torch.randn(H, generator=g) if norm else None
    f = torch.tensor([10000.0 ** (-2.0 * i / H) for i in range((H + 1) // 2)], dtype=torch.float64)
    h, x = k_.embed_sinusoid(ids.to(DEV), pos.to(DEV), table.to(DEV), 1.3, k_.rotary_table(f).to(DEV),
                             w.to(DEV) if norm else None, 1e-5, dt)
    a = pos.double()[:, None] * f[None, :]
    want = torch.stack([a.sin(), a.cos()], dim=-1).reshape(len(pos), -1)[:, :H] + 1.3 * table[ids.long()].double()
    if norm:
        want = want / torch.sqrt((want * want).mean(-1, keepdim=True) + 1e-5) * w.double()
    close(h, want, torch.float32)
    if dt == torch.bfloat16:
        assert torch.equal(x, h.bfloat16())
    else:
        assert x is None


@pytest.mark.parametrize("dt", TYPES)
@pytest.mark.parametrize("x_dt", TYPES)
@pytest.mark.parametrize("H, G, d, dv, row, temp", [
    (4, 2, 24, 16, 0, (0.5, 10)), (3, 1, 10, 6, 0, None), (6, 3, 16, 40, 64, (0.2, 1)), (12, 4, 64, 48, 64, (-0.1, 64)),
    (40, 8, 64, 64, 64, (0.3, 7)), (5, 5, 12, 90, 128, (0.1, 1000)), (2, 1, 136, 120, 0, (0.4, 2.5))])
def test_one_norm_over_all_heads_and_a_temperature(dt, x_dt, H, G, d, dv, row, temp):
    """Queries and keys normed over all their heads together, the queries' temperature, rows padded to ``row`` in the cache
    and for the queries; and a layer with queries only.  More heads than a block takes, of which some hold queries only,
    keys only, or both."""
    g = torch.Generator().manual_seed(2)
    k_ = K()
    page, n_pages = 64, 8
    dp, dvp = (row or (d + 7) // 8 * 8), (row or (dv + 7) // 8 * 8)
    tok_seq = torch.tensor([0] * 9 + [1] * 3 + [2] * 2, dtype=torch.int32)
    tok_pos = torch.tensor(list(range(60, 69)) + [0, 1, 2] + [130, 131], dtype=torch.int32)
    T = len(tok_pos)
    for off, ld_mod in ((8, 8), (5, 1)):
        ld = (off + (H + G) * d + G * dv + 3 + ld_mod - 1) // ld_mod * ld_mod
        x = torch.randn(T, ld, generator=g).to(x_dt)
        qw, kw = 1 + 0.3 * torch.randn(H * d, generator=g), 1 + 0.3 * torch.randn(G * d, generator=g)
        bt = torch.tensor([[4, 1, -1], [0, -1, -1], [3, 5, 2]], dtype=torch.int32)
        kp = torch.full((n_pages, G, page, dp), 7.0, dtype=dt, device=DEV)
        vp = torch.full((n_pages, G, page, dvp), 7.0, dtype=dt, device=DEV)
        args = (1e-5, 0, 0, None, 1.0, 1.0, None, tok_pos.to(DEV), tok_seq.to(DEV), bt.to(DEV), page, dt)
        q, none = k_.qk_prep(x.to(DEV), off, off + H * d, off + (H + G) * d, H, G, d, dv, dp, dvp, 3, qw.to(DEV), kw.to(DEV),
                             *args, kp, vp, temperature=temp)
        assert none is None
        xd = x.double()
        nrm = lambda a, w: a / torch.sqrt((a * a).mean(-1, keepdim=True) + 1e-5) * w.double()
        qr = nrm(xd[:, off:off + H * d], qw)
        if temp:
            qr = qr * torch.tensor([1 + temp[0] * math.log(math.floor((int(p) + 1) / temp[1]) + 1) for p in tok_pos],
                                   dtype=torch.float64)[:, None]
        kr = nrm(xd[:, off + H * d:off + (H + G) * d], kw).reshape(T, G, d)
        vr = xd[:, off + (H + G) * d:off + (H + G) * d + G * dv].reshape(T, G, dv)
        want_q = torch.zeros(T, H, dp, dtype=torch.float64)
        want_q[..., :d] = qr.reshape(T, H, d)
        close(q.reshape(T, H, dp), want_q, dt, "q")
        want_k, want_v = torch.full(kp.shape, 7.0, dtype=torch.float64), torch.full(vp.shape, 7.0, dtype=torch.float64)
        for t in range(T):
            p = int(tok_pos[t])
            pg = int(bt[int(tok_seq[t]), p // page])
            want_k[pg, :, p % page, :] = 0
            want_v[pg, :, p % page, :] = 0
            want_k[pg, :, p % page, :d] = kr[t]
            want_v[pg, :, p % page, :dv] = vr[t]
        close(kp, want_k, dt, "keys, and no other place of the pool")
        close(vp, want_v, dt, "values, and no other place of the pool")
        # queries only, of the same columns: the same numbers
        q2, _ = k_.qk_prep(x.to(DEV), off, 0, -1, H, 0, d, dv, dp, dvp, 3, qw.to(DEV), None, *args, None, None, temperature=temp)
        close(q2.reshape(T, H, dp), want_q, dt, "queries only")


class Case:
    """Sequences over shuffled pages, queries of one token each, score biases by distance and a sink per head."""

    def __init__(self, H, G, d, dv, near, dt, queries, lens=(700, 1, 130, 65), seed=4):
        g = torch.Generator().manual_seed(seed)
        self.page, n_pages, width = 64, 40, 12
        self.H, self.G, self.d, self.dv = H, G, d, dv
        perm = torch.randperm(n_pages, generator=g)
        bt = torch.full((len(lens), width), -1, dtype=torch.int32)
        at = 0
        for b, n in enumerate(lens):
            need = (n + 63) // 64
            bt[b, :need] = perm[at:at + need].int()
            at += need
        kp = torch.randn(n_pages, G, 64, d, generator=g).to(dt)
        vp = torch.randn(n_pages, G, 64, dv, generator=g).to(dt)
        self.T = len(queries)
        q = torch.randn(self.T, H * d, generator=g).to(dt)
        bias = 3.0 * torch.randn(H, near, generator=g)
        sink = 3.0 * torch.rand(H, generator=g) - 1.0
        self.scale = 0.9 / math.sqrt(d)
        want = torch.zeros(self.T, H, dv, dtype=torch.float64)
        for t, (b, p) in enumerate(queries):
            js = torch.arange(p + 1)
            pg = bt[b, js // 64].long()
            kk, vv = kp[pg, :, js % 64].double(), vp[pg, :, js % 64].double()
            back = p - js
            for h in range(H):
                s = kk[:, h // (H // G)] @ q[t, h * d:(h + 1) * d].double() * self.scale
                s = s + torch.where(back < near, bias[h, back.clamp(max=near - 1)].double(), torch.zeros((), dtype=torch.float64))
                m = float(s.max())
                e = torch.exp(s - m)
                want[t, h] = (e / (e.sum() + math.exp(float(sink[h]) - m))) @ vv[:, h // (H // G)]
        self.want = want
        self.q, self.kp, self.vp, self.bt = q.to(DEV), kp.to(DEV), vp.to(DEV), bt.to(DEV)
        self.tok_seq = torch.tensor([b for b, _ in queries], dtype=torch.int32, device=DEV)
        self.tok_pos = torch.tensor([p for _, p in queries], dtype=torch.int32, device=DEV)
        self.dist, self.sink = K().distance_table(bias).to(DEV), sink.to(DEV)


@pytest.mark.parametrize("dt", TYPES)
@pytest.mark.parametrize("H, G, d, dv, near", [(4, 2, 24, 16, 50), (6, 2, 16, 40, 1), (2, 1, 64, 64, 300), (3, 3, 16, 8, 64),
                                               (20, 1, 16, 16, 129), (5, 5, 160, 136, 1000)])
def test_distance_biases_on_the_cuda_cores(dt, H, G, d, dv, near):
    queries = [(0, 699), (0, 450), (0, 256), (0, 255), (0, 0), (1, 0), (2, 129), (2, 127), (2, 128), (3, 64), (3, 63),
               (0, min(near, 699)), (0, min(near - 1, 699)), (0, min(near + 63, 699))]
    c = Case(H, G, d, dv, near, dt, queries)
    k_ = K()
    for split in (256, 64):
        n = (700 + split - 1) // split
        for T in (c.T, 2):                             # two tokens: the merge inside the attention kernel
            scratch = torch.zeros(k_.attn_tokens_scratch_bytes(T, H, dv, n) // 4 + 1, device=DEV)
            out = torch.empty(T, H * dv, dtype=dt, device=DEV)
            k_.attn_tokens_ex(c.q[:T], H * d, out, c.kp, c.vp, c.bt, c.tok_pos[:T], c.tok_seq[:T], T, H, G, d, dv, 64, 0, 0, True,
                              c.scale, split, n, scratch, sink_vals=c.sink, dist=c.dist)
            close(out.reshape(T, H, dv), c.want[:T], dt, f"split {split}, {T} tokens")


@pytest.mark.parametrize("H, G, d, near", [(4, 2, 64, 50), (8, 1, 128, 300), (12, 1, 64, 1), (4, 4, 128, 65), (32, 2, 64, 128),
                                           (6, 2, 64, 900)])
def test_distance_biases_and_sinks_for_single_tokens(H, G, d, near):
    """The decode kernel's ways of ending a row (one chunk; chunks merged through scratch; inside a block or a cluster), with
    groups of heads split and in twins."""
    queries = [(0, 699), (1, 0), (2, 129), (3, 64), (0, min(near, 699)), (0, min(near - 1, 699)), (0, 448), (0, 447)]
    c = Case(H, G, d, d, near, torch.bfloat16, queries)
    k_ = K()
    group = H // G
    for split, in_block, head_split, twins in ((1024, 0, 1, 1), (256, 0, 1, 1), (64, 0, 2, 1), (256, 1, 1, 1), (128, 2, 1, 1),
                                               (256, 1, 2, 2), (128, 2, 2, 2)):
        if group % head_split or (twins == 2 and group // head_split > 8):
            continue
        n = (700 + split - 1) // split
        scratch = torch.zeros(k_.attn_tokens_scratch_bytes(c.T, H, d, n) // 4 + 1, device=DEV) if n > 1 and not in_block else None
        out = torch.empty(c.T, H * d, dtype=torch.bfloat16, device=DEV)
        k_.attn_decode(c.q, H * d, out, c.kp, c.vp, c.bt, c.tok_pos, c.tok_seq, c.T, H, G, d, 64, 0, c.scale, split, n, scratch,
                       in_block=in_block, head_split=head_split, twins=twins, sink=True, sink_vals=c.sink, dist=c.dist)
        close(out.reshape(c.T, H, d), c.want, torch.bfloat16, f"split {split} in_block {in_block} heads / {head_split}")
    assert k_.attn_decode_status() == 0


def test_decode_kernel_biases_the_key_it_takes_from_the_projection():
    """With the token's own key and value out of the projection's row: distance zero has its bias."""
    H, G, d = 4, 2, 64
    c = Case(H, G, d, d, 40, torch.bfloat16, [(0, 699), (2, 129)], seed=6)
    k_ = K()
    rows = []
    for t in range(2):
        b, p = int(c.tok_seq[t]), int(c.tok_pos[t])
        pg = int(c.bt[b, p // 64])
        rows.append(torch.cat([c.q[t], c.kp[pg, :, p % 64].reshape(-1), c.vp[pg, :, p % 64].reshape(-1)]))
        c.kp[pg, :, p % 64] = 9.0                     # the kernel must put the key and the value here itself
        c.vp[pg, :, p % 64] = 9.0
    qkv = torch.stack(rows).contiguous()
    scratch = torch.zeros(k_.attn_tokens_scratch_bytes(2, H, d, 3) // 4 + 1, device=DEV)
    out = torch.empty(2, H * d, dtype=torch.bfloat16, device=DEV)
    k_.attn_decode(qkv, qkv.stride(0), out, c.kp, c.vp, c.bt, c.tok_pos, c.tok_seq, 2, H, G, d, 64, 0, c.scale, 256, 3, scratch,
                   write_new=True, sink=True, sink_vals=c.sink, dist=c.dist)
    close(out.reshape(2, H, d), c.want, torch.bfloat16)


@pytest.mark.parametrize("nh, nkv, hd", [(4, 2, 64), (8, 1, 64), (4, 2, 128), (5, 1, 128)])
@pytest.mark.parametrize("near, cap, window", [(50, 0.0, 0), (1, 0.0, 0), (130, 9.0, 0), (600, 0.0, 0), (64, 0.0, 100)])
def test_distance_biases_for_prompts(nh, nkv, hd, near, cap, window):
    """Whole prompts, portions after earlier context and single rows through the tcgen05 kernel in each of its forms: biases
    shorter than a page, over several pages and over everything, with a sink per head, after a cap, under a window."""
    from test_kernels_gpu import PagedCase
    k_ = K()
    case = PagedCase(lens=[300, 64, 1, 700, 65, 128, 129], new=[300, 64, 1, 200, 65, 1, 129], nh=nh, nkv=nkv, hd=hd,
                     dtype=torch.bfloat16, seed=hd + nh + near)
    T = case.q.shape[0]
    buf = case.q.reshape(T, nh * hd).to(DEV).contiguous()
    scale = 1.3 / math.sqrt(hd)
    g = torch.Generator().manual_seed(3)
    sink = 3.0 * torch.rand(nh, generator=g) - 1.0
    bias = 3.0 * torch.randn(nh, near, generator=g)
    outs, t, G = [], 0, nh // nkv
    for b, (n, m) in enumerate(zip(case.lens, case.new)):
        k, v = (a[b].double().repeat_interleave(G, dim=1) for a in (case.k, case.v))
        s = torch.einsum("qhd,khd->hqk", case.q[t:t + m].double(), k) * scale
        if cap:
            s = cap * torch.tanh(s / cap)
        back = torch.arange(n - m, n)[:, None] - torch.arange(n)[None, :]
        s = s + torch.where((back >= 0) & (back < near), bias.double()[:, back.clamp(0, near - 1)], torch.zeros((), dtype=torch.float64))
        s = s.masked_fill((back < 0) | ((back >= window) if window else (back < 0)), float("-inf"))
        mx = s.max(dim=-1, keepdim=True).values
        e = torch.exp(s - mx)
        outs.append(torch.einsum("hqk,khd->qhd", e / (e.sum(-1, keepdim=True) + torch.exp(sink.double()[:, None, None] - mx)), v))
        t += m
    want = torch.cat(outs).reshape(-1, nh * hd)
    tile_seq, tile_q0 = case.tiles(128)
    got = []
    for variant in ((0, 1, 2, 3) if hd == 64 else (0, 1, 3)):
        o = torch.full((T, nh * hd), 3.0, device=DEV, dtype=torch.bfloat16)
        k_.attn_prefill_tc(buf, buf.stride(0), o, case.k_pool, case.v_pool, case.table, case.row_start, case.row_pos0,
                           tile_seq, tile_q0, tile_seq.numel(), nh, nkv, hd, 64, window, scale, variant=variant, sink=True,
                           softcap=cap, sink_vals=sink.to(DEV), dist=k_.distance_table(bias).to(DEV))
        err = float((o.double().cpu() - want).abs().max()) / float(want.abs().max())
        assert err <= 1e-2, (variant, err)
        got.append(o)
    for o in got[1:]:
        assert torch.equal(got[0], o)
    assert k_.attn_prefill_tc_status() == 0


@pytest.mark.parametrize("dt", TYPES)
@pytest.mark.parametrize("T, W, n, top", [(1, 96, 8, 2), (5, 100, 12, 12), (37, 2048, 64, 6), (150, 1100, 9, 3), (3, 72, 1, 1)])
def test_choice_by_biased_logits(dt, T, W, n, top):
    """Logits far from zero, a bias that changes choices, weights that are the softmax over the picks alone."""
    g = torch.Generator().manual_seed(T + W + n)
    x = torch.randn(T, W, generator=g).to(dt)
    wr = torch.randn(n, W, generator=g) * 3.0 / math.sqrt(W)
    bias = 2.0 * torch.randn(n, generator=g) - 60.0       # far below: plain exponentials of these would vanish
    idx, wt, gate = K().moe_route(x.to(DEV), wr.to(DEV), bias.to(DEV), n, 0, 1, 1, top, 1.5, "picked")
    z = x.double() @ wr.double().T + bias.double()
    best = torch.sort(z, dim=-1, descending=True)
    assert gate is None and idx.cpu().tolist() == best.indices[:, :top].tolist()
    close(wt, 1.5 * torch.softmax(best.values[:, :top], dim=-1), torch.float32)
    if T > 64:
        idx1, wt1, _ = K().moe_route(x[:3].to(DEV), wr.to(DEV), bias.to(DEV), n, 0, 1, 1, top, 1.5, "picked")
        assert torch.equal(idx1, idx[:3]) and torch.equal(wt1, wt[:3])


def test_squared_relu_experts():
    """The three products of the experts with squared relu between them."""
    g = torch.Generator().manual_seed(9)
    k_ = K()
    for kind, T, dt in (("tile", 20, torch.float32), ("tile", 70, torch.bfloat16), ("few", 6, torch.bfloat16), ("tc", 400, torch.bfloat16)):
        top, E, W, inner = 2, 5, 96, 72
        x = torch.randn(T, W, generator=g).to(dt)
        idx = torch.randint(0, E, (T, top), generator=g, dtype=torch.int32)
        w = (torch.randn(E, inner, W, generator=g) / math.sqrt(W)).to(dt)
        want = torch.stack([torch.relu(w[int(idx[p // top, p % top])].double() @ x[p // top].double()) ** 2 for p in range(T * top)])
        order, plan = k_.moe_plan(idx.to(DEV), E, k_.moe_tile_rows(kind))
        if kind == "tc":
            mid = k_.moe_gemm_tc(k_.moe_gather(x.to(DEV), top, order, plan), w.to(DEV), order, plan, dt, act="relu2")
            want = want[order.long().cpu()]
        else:
            mid = (k_.moe_gemm if kind == "tile" else k_.moe_gemv)(x.to(DEV), top, w.to(DEV), order, plan, dt, act="relu2")
        close(mid, want, dt, kind)
    assert k_.moe_tc_status() == 0


@pytest.mark.parametrize("s_dt", TYPES)
@pytest.mark.parametrize("H, top, with_shared, with_gate", [(96, 2, True, False), (100, 3, False, False), (8192, 1, True, True),
                                                            (2304, 4, True, False)])
def test_weighted_sum_and_its_norm_in_one_kernel(s_dt, H, top, with_shared, with_gate):
    g = torch.Generator().manual_seed(H)
    k_ = K()
    T, E = 7, 5
    y = torch.randn(T * top, H, generator=g)
    idx = torch.randint(0, E, (T, top), generator=g, dtype=torch.int32)
    wt = torch.rand(T, top, generator=g)
    shared = torch.randn(T, H, generator=g).to(s_dt) if with_shared else None
    gate = torch.rand(T, generator=g) if with_gate else None
    h0, w = torch.randn(T, H, generator=g), 1.0 + 0.2 * torch.randn(H, generator=g)
    v = torch.einsum("tk,tkh->th", wt.double(), y.double().reshape(T, top, H))
    if with_shared:
        v = v + shared.double() * (gate.double()[:, None] if with_gate else 1.0)
    want = h0.double() + v / torch.sqrt((v * v).mean(-1, keepdim=True) + 1e-5) * w.double()
    for want_x in (True, False):
        h = h0.clone().to(DEV)
        x = k_.moe_combine_norm(y.to(DEV), idx.to(DEV), wt.to(DEV), shared.to(DEV) if with_shared else None,
                                gate.to(DEV) if with_gate else None, E, h, w.to(DEV), 1e-5, want_x)
        close(h, want, torch.float32)
        assert (x is None) if not want_x else torch.equal(x, h.bfloat16())
