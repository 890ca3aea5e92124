"""The kernels that the Korazen design added or widened, each alone against a float64 restatement of its own operation
written here: the embedding's normed rows, branches joining the stream (one, or two that are normed first), columns handed
from one product to another, the clamped gated activation in every product's epilogue and apart, weighted unit norms per
head, attention whose values have another size than its keys (blocks, page borders, a key that outweighs all others just
inside and just outside a block), and the gated delta rule (whole, in pieces, token by token, batches of unequal sequences,
key heads shared by value heads, decays of exactly one and of zero, a write that must be read back after hundreds of tokens)."""
import numpy as np
import pytest
import torch

from test_gpu_lavutar_kernels import BF16_ULP, DEV, Pages, _blocks, _close, _i32, _ops, _rand

pytestmark = pytest.mark.gpu

TOL = {torch.float32: (3e-6, 0.0), torch.bfloat16: (1.5 * BF16_ULP, BF16_ULP)}


def _rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def _d(x):
    return x.double().cpu()


# ------------------------------------------------------------------ the stream

@pytest.mark.parametrize("table_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("D", [1, 44, 192, 1000, 4100, 9000])
def test_embedding_rows_are_normed_on_their_way(D, table_dtype):
    ops = _ops()
    table, gain, toks = _rand((50, D), table_dtype, 1, 3.0), _rand((D,), torch.float32, 2) + 1.0, [3, 49, 0, 3]
    ref = _rms(_d(table)[toks], 1e-5) * _d(gain)
    for rows_dtype in (None, torch.float32, torch.bfloat16):
        x, rows = ops.embedding_norm(table, _i32(toks), gain, 1e-5, rows_dtype)
        _close(x, ref, 3e-6)
        if rows_dtype is None:
            assert rows is None
        else:
            assert torch.equal(rows, x.to(rows_dtype))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("D", [1, 44, 190, 192, 1000, 2048, 4100, 9000])
def test_branches_join_the_stream_behind_their_norms(D, dtype):
    ops = _ops()
    T, eps, eps_in = 5, 1e-5, 1e-6
    y1, y2, x0 = _rand((T, D), torch.float32, 1, 0.01), _rand((T, D), torch.float32, 2, 30.0), _rand((T, D), torch.float32, 3)
    b1, w1, w2, gain, nxt = (_rand((D,), torch.float32, s) + o for s, o in ((4, 0.0), (5, 1.0), (6, 1.0), (7, 1.0), (8, 1.0)))
    one = _d(x0) + _rms(_d(y1) + _d(b1), eps) * _d(gain)
    plain = _d(x0) + _rms(_d(y1), eps) * _d(gain)
    both = 0.5 * _rms(_d(y1) + _d(b1), eps_in) * _d(w1) + 0.5 * _rms(_d(y2), eps_in) * _d(w2)
    two = _d(x0) + _rms(both, eps) * _d(gain)
    for branches, ref in ((((y1, b1),), one), (((y1, None),), plain), (((y1, b1, w1, 0.5), (y2, None, w2, 0.5), eps_in), two)):
        x = x0.clone()
        assert ops.join_normed(x, branches, gain, eps) is None
        _close(x, ref, 1e-5)
        x = x0.clone()
        rows = ops.join_normed(x, branches, gain, eps, dtype)
        assert torch.equal(rows, x.to(dtype))                     # the stream as the next sublayer reads it
        _close(x, ref, 1e-5)
        x = x0.clone()
        rows = ops.join_normed(x, branches, gain, eps, dtype, next_norm=(nxt, 1e-4))
        _close(rows, _rms(ref, 1e-4) * _d(nxt), 2e-5 if dtype == torch.float32 else TOL[dtype][0], TOL[dtype][1])


def test_columns_go_to_another_product_whole_or_in_two_terms():
    ops = _ops()
    rows = _rand((9, 61), torch.float32, 1, 5.0)
    for dtype in (torch.float32, torch.bfloat16):
        out = ops.take_columns(rows, 17, 21, 24, dtype)
        assert torch.equal(out[:, :21], rows[:, 17:38].to(dtype)) and float(out[:, 21:].abs().max()) == 0.0
    out = ops.take_columns(rows, 17, 21, 24, torch.bfloat16, split=True)
    assert out.shape == (9, 48) and torch.equal(out[:, :21], rows[:, 17:38].to(torch.bfloat16))
    both = _d(out[:, :24]) + _d(out[:, 24:])
    assert float(((both[:, :21] - _d(rows[:, 17:38])).abs() / _d(rows[:, 17:38]).abs()).max()) < 2.0 ** -16
    assert ops.stream_rows(rows, torch.float32) is rows and torch.equal(ops.stream_rows(rows, torch.bfloat16), rows.to(torch.bfloat16))


# ------------------------------------------------------------------ the clamped gated activation

def _clamped(g, u, limit):
    g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1.0)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("limit", [0.7, 7.0])
@pytest.mark.parametrize("F", [24, 37])
def test_clamped_activation_apart(dtype, limit, F):
    ops = _ops()
    gu, bias = _rand((7, 2 * F), dtype, 1, 3.0), _rand((2 * F,), torch.float32, 2)
    g, u = _d(gu)[:, :F], _d(gu)[:, F:]
    _close(ops.swiglu(gu, 0, limit=limit), _clamped(g, u, limit), *TOL[dtype])
    _close(ops.gated_act(gu, None, "sigmoid_clamped", dtype, limit), _clamped(g, u, limit), *TOL[dtype])
    _close(ops.gated_act(gu, bias, "sigmoid_clamped", dtype, limit), _clamped(g + _d(bias)[:F], u + _d(bias)[F:], limit), *TOL[dtype])


@pytest.mark.parametrize("M,F,K", [(1, 40, 64), (8, 320, 192), (16, 64, 256), (17, 512, 256), (64, 3000, 64), (100, 48, 640), (300, 1024, 128),
                                   (700, 4096, 256), (130, 44, 64)])
@pytest.mark.parametrize("limit", [0.0, 1.2])
def test_clamped_activation_in_the_products_epilogues(M, F, K, limit):
    """Rows for every kernel of the choice: streamed weights, tcgen05 tiles (whole and with the contraction cut), pairs of
    multiprocessors.  limit 0 is the plain form."""
    from longbow_quarrel_b200.kernels import linear
    x, gate, up = _rand((M, K), torch.bfloat16, 1), _rand((F, K), torch.bfloat16, 2, 2.0 * K ** -0.5), _rand((F, K), torch.bfloat16, 3, 2.0 * K ** -0.5)
    block = linear.GATE_UP_BLOCK if F % 8 == 0 else 0
    w = linear.LinearWeight(linear.interleave_gate_up(gate, up) if block else torch.cat([gate, up]))
    got = linear.linear_swiglu(x, w, block, limit)
    g, u = _d(x) @ _d(gate).T, _d(x) @ _d(up).T
    ref = _clamped(g, u, limit) if limit else u * g * torch.sigmoid(g)
    # (without a block the halves are rounded to bfloat16 before the activation)
    _close(got, ref, (3 if block else 10) * BF16_ULP, BF16_ULP)


# ------------------------------------------------------------------ weighted unit norms per head

@pytest.mark.parametrize("in_dtype,out_dtype", [(torch.float32, torch.float32), (torch.float32, torch.bfloat16)])
@pytest.mark.parametrize("H,G,hd,vd,rot", [(4, 2, 32, 48, 16), (3, 1, 26, 12, 0), (2, 2, 64, 64, 64)])
def test_weighted_unit_norms_behind_the_bias_and_ahead_of_the_rotation(in_dtype, out_dtype, H, G, hd, vd, rot):
    ops = _ops()
    page, eps = 64, 1e-5
    tok_pos, tok_seq = [0, 1, 63, 64, 130], [0, 0, 0, 0, 1]
    T, width = len(tok_pos), (H + G) * hd + G * vd
    src, bias = _rand((T, width), in_dtype, 1), _rand((width,), torch.float32, 2)
    wq, wk = _rand((hd,), torch.float32, 3) + 1.0, _rand((hd,), torch.float32, 4) + 1.0
    weight = torch.cat([wq.repeat(H), wk.repeat(G)]).contiguous()
    ang = torch.arange(200, dtype=torch.float64)[:, None] * torch.rand(max(rot // 2, 1), dtype=torch.float64)[None, :]
    cos, sin = torch.cos(ang).float().to(DEV), torch.sin(ang).float().to(DEV)
    table = torch.tensor([[2, 0, 4], [1, 3, 5]], dtype=torch.int32, device=DEV)
    k_pages = torch.zeros((6, G, page, hd), dtype=out_dtype, device=DEV)
    v_pages = torch.zeros((6, G, page, vd), dtype=out_dtype, device=DEV)
    q_out = torch.empty((T, H * hd), dtype=out_dtype, device=DEV)
    ops.rope_partial(src, bias, cos if rot else None, sin if rot else None, rot, _i32(tok_pos), _i32(tok_seq), _i32([0, 1]), table, k_pages,
                     v_pages, H + G, H, G, hd, vd, (H + G) * hd, page, qout=q_out, unit_norm="head", norm_weight=weight, norm_eps=eps)
    x = _d(src) + _d(bias)
    heads = _rms(x[:, :(H + G) * hd].reshape(T, H + G, hd), eps)
    heads[:, :H] *= _d(wq)
    heads[:, H:] *= _d(wk)
    if rot:
        c, s, half = _d(cos)[tok_pos][:, None], _d(sin)[tok_pos][:, None], rot // 2
        a, b = heads[..., :half].clone(), heads[..., half:rot].clone()
        heads[..., :half], heads[..., half:rot] = a * c - b * s, b * c + a * s
    tol = TOL[out_dtype]
    _close(q_out.reshape(T, H, hd), heads[:, :H], *tol)
    for r, (p, b) in enumerate(zip(tok_pos, tok_seq)):
        pg = int(table[b, p // page])
        _close(k_pages[pg, :, p % page], heads[r, H:], *tol)
        _close(v_pages[pg, :, p % page], x[r, (H + G) * hd:].reshape(G, vd), *tol)


# ------------------------------------------------------------------ values of another size than keys

# H, G, hd, vd, block
SIZES = [(9, 3, 112, 224, 90), (4, 2, 16, 32, 37), (8, 2, 64, 128, 64), (3, 1, 128, 256, 100), (4, 4, 128, 40, None), (2, 1, 48, 160, 1),
         (20, 1, 32, 64, 200), (2, 2, 80, 24, 70)]


@pytest.mark.parametrize("H,G,hd,vd,block", SIZES)
def test_decode_attention_with_values_of_another_size(H, G, hd, vd, block):
    """One token per sequence at its end, in equal slices and from work lists; the pages below its block are gone."""
    ops = _ops()
    from longbow_quarrel_b200.kernels.attention import MAX_SPLITS, cut_decode_work
    lens = [300, 1, 77, 64, 17, 1500, 33, 201, 200]
    tok_pos, tok_seq = [n - 1 for n in lens], list(range(len(lens)))
    case = Pages(lens, G, hd, vd, torch.bfloat16, seed=3, block=block, first_query=tok_pos)
    q = _rand((len(lens), H * hd + 8 * G), torch.bfloat16, 71)
    scale = 0.9 * hd ** -0.5
    ref = case.reference(q[:, :H * hd].reshape(-1, H, hd), tok_seq, tok_pos, H, scale, block)
    args = (q, case.k_pages, case.v_pages, case.table, _i32(tok_pos), _i32(tok_seq), case.slots, H, G, hd, case.page, scale, ops.span(None, block))
    for splits in (1, 3):
        _close(ops.attn_decode(*args, splits, vd=vd).reshape(-1, H, vd), ref, case.tol(ref), BF16_ULP)
    for teams in (9, 40):
        work = cut_decode_work(tok_pos, 0, teams, chunk=block or 0)
        out = ops.attn_decode(*args, min(MAX_SPLITS, teams), early_loads=True, work=_i32(work.tolist()), teams=teams, vd=vd)
        _close(out.reshape(-1, H, vd), ref, case.tol(ref), BF16_ULP)


@pytest.mark.parametrize("H,G,hd,vd,block", SIZES)
def test_prompt_attention_with_values_of_another_size(H, G, hd, vd, block):
    """One sequence whole from its first token, one single token, one that goes on after 270 cached tokens."""
    ops = _ops()
    lens, new, past = [300, 1, 400], [300, 1, 130], [0, 0, 270]
    case = Pages(lens, G, hd, vd, torch.bfloat16, seed=5, block=block, first_query=past)
    tok_seq = [b for b, n in enumerate(new) for _ in range(n)]
    tok_pos = [p + i for n, p in zip(new, past) for i in range(n)]
    q = _rand((sum(new), H * hd), torch.bfloat16, 73)
    scale = hd ** -0.5
    ref = case.reference(q.reshape(-1, H, hd), tok_seq, tok_pos, H, scale, block)
    out = ops.attn_prefill(q, case.k_pages, case.v_pages, case.table, case.slots, _i32(lens), _blocks(new, past, 64), H, G, hd, case.page, scale,
                           ops.span(None, block), vd=vd)
    _close(out.reshape(-1, H, vd), ref, case.tol(ref), BF16_ULP)


@pytest.mark.parametrize("kernel", ["prefill", "decode"])
@pytest.mark.parametrize("hd,vd,block", [(64, 128, 60), (80, 160, 64), (128, 48, 100), (32, 64, 7)])
def test_one_key_that_outweighs_all_others_shows_a_block_s_edges(kernel, hd, vd, block):
    """A key aimed at every query stands at a block's first place, at its last, and at the place before it: positions of the
    block see exactly that key's value, positions outside it nothing of it."""
    ops = _ops()
    n, scale = 3 * block + 5, 1.0
    q = torch.ones((n, hd), dtype=torch.bfloat16, device=DEV)
    for at in (block, 2 * block - 1, block - 1):
        case = Pages([n], 1, hd, vd, torch.bfloat16, seed=at)
        case.plant(0, at, 2.0)                                    # its score exceeds every other by far
        args = (case.k_pages, case.v_pages, case.table)
        if kernel == "decode":
            out = torch.cat([ops.attn_decode(q[p:p + 1], *args, _i32([p]), _i32([0]), case.slots, 1, 1, hd, 64, scale, -block, 2, vd=vd) for p in range(n)])
        else:
            out = ops.attn_prefill(q, *args, case.slots, _i32([n]), _blocks([n], [0], 64), 1, 1, hd, 64, scale, -block, vd=vd)
        want = case.v[0][at, 0].double().cpu()
        for p in range(n):
            same = float((out[p].double().cpu() - want).abs().max()) < 2e-2 * float(want.abs().max())
            assert same == (p >= at and p // block == at // block), (at, p)


# ------------------------------------------------------------------ the gated delta rule

class Delta:
    """Random rows of sequences, and the rule in float64 with the state and the convolution's past carried by hand."""

    def __init__(self, H, G, dk, dv, taps, lens, seed, ra=5, rg=7, rate=None, bias=None):
        self.H, self.G, self.dk, self.dv, self.taps, self.ra, self.rg = H, G, dk, dv, taps, ra, rg
        self.C = 2 * G * dk + H * dv
        self.b_off, self.a_off = self.C, self.C + H
        self.g_off = self.a_off + ra
        self.rows = [_rand((n, self.g_off + rg), torch.float32, seed * 10 + i) for i, n in enumerate(lens)]
        self.taps_w = _rand((taps, self.C), torch.float32, seed + 900, 0.6)
        self.ra_ld, self.rg_ld = -(-ra // 8) * 8, -(-rg // 8) * 8
        self.a2 = torch.nn.functional.pad(_rand((H * dk, ra), torch.bfloat16, seed + 901, 0.7), (0, self.ra_ld - ra)).contiguous()
        self.g2 = torch.nn.functional.pad(_rand((H * dv, rg), torch.bfloat16, seed + 902), (0, self.rg_ld - rg)).contiguous()
        self.bias = _rand((H * dk,), torch.float32, seed + 903) - 2.0 if bias is None else torch.full((H * dk,), bias, device=DEV)
        self.rate = torch.exp(_rand((H,), torch.float32, seed + 904)) if rate is None else torch.full((H,), rate, device=DEV)
        self.norm_w = _rand((dv,), torch.float32, seed + 905) + 1.0
        n_slots = len(lens) + 3
        self.slot_of = [int(s) for s in np.random.default_rng(seed).permutation(n_slots)[:len(lens)]]
        self.state = torch.zeros((n_slots, H, dk, dv), dtype=torch.float32, device=DEV)
        self.ring = torch.full((n_slots, taps, self.C), 77.0, dtype=torch.float32, device=DEV)   # rows ahead of a sequence must not be read

    def z(self, rows):
        return (rows[:, self.a_off:self.a_off + self.ra].double() @ self.a2[:, :self.ra].double().T).float().contiguous()

    def reference(self, i):
        """(o [n, H, dv], S) of sequence i."""
        x = _d(self.rows[i])
        n, H, G, dk, dv = x.shape[0], self.H, self.G, self.dk, self.dv
        w = _d(self.taps_w)
        y = torch.zeros(n, self.C, dtype=torch.float64)
        for j in range(self.taps):
            back = self.taps - 1 - j
            if back < n:
                y[back:] += w[j] * x[:n - back, :self.C]
        y = y * torch.sigmoid(y)
        q, k, v = y[:, :G * dk].reshape(n, G, dk), y[:, G * dk:2 * G * dk].reshape(n, G, dk), y[:, 2 * G * dk:].reshape(n, H, dv)
        q = q / torch.sqrt((q * q).sum(-1, keepdim=True) + 1e-6) * dk ** -0.5
        k = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
        q, k = q.repeat_interleave(H // G, 1), k.repeat_interleave(H // G, 1)
        b = torch.sigmoid(x[:, self.b_off:self.b_off + H])
        z = x[:, self.a_off:self.a_off + self.ra] @ _d(self.a2)[:, :self.ra].T + _d(self.bias)
        a = torch.exp(-_d(self.rate)[None, :, None] * torch.nn.functional.softplus(z).reshape(n, H, dk))
        S, o = torch.zeros(H, dk, dv, dtype=torch.float64), torch.zeros(n, H, dv, dtype=torch.float64)
        for t in range(n):
            S = a[t][:, :, None] * S
            u = b[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
            S = S + k[t][:, :, None] * u[:, None, :]
            o[t] = torch.einsum("hdv,hd->hv", S, q[t])
        return o, S

    def step(self, takes):
        """takes: (sequence, first row, rows) for each of the step's sequences; raw outputs in that order."""
        rows = torch.cat([self.rows[i][lo:lo + n] for i, lo, n in takes]).contiguous()
        cu = np.cumsum([0] + [n for _, _, n in takes]).tolist()
        pos = [lo + t for _, lo, n in takes for t in range(n)]
        return _ops().delta_prompt(rows, self.b_off, self.taps_w, self.ring, self.z(rows), self.bias, self.rate, self.state, _i32(cu),
                                   _i32([self.slot_of[i] for i, _, _ in takes]), _i32(pos), len(takes), max(n for _, _, n in takes), self.H, self.G,
                                   self.dk, self.dv, self.dk ** -0.5, 1e-6)

    def single(self, takes, dtype):
        """takes: (sequence, row): one token each, normed and gated."""
        rows = torch.cat([self.rows[i][t:t + 1] for i, t in takes]).contiguous()
        return _ops().delta_single(rows, self.b_off, self.taps_w, self.ring, self.bias, self.rate, self.state, _i32(list(range(len(takes) + 1))),
                                   _i32([self.slot_of[i] for i, _ in takes]), _i32([t for _, t in takes]), self.a_off, self.ra, self.a2, self.g_off,
                                   self.rg, self.g2, self.norm_w, 1e-5, dtype, len(takes), self.H, self.G, self.dk, self.dv, self.dk ** -0.5, 1e-6)

    def finished(self, i, o):
        """What the single-token kernel makes of raw outputs o [n, H, dv] of sequence i."""
        gate = torch.sigmoid(_d(self.rows[i])[:, self.g_off:self.g_off + self.rg] @ _d(self.g2)[:, :self.rg].T)
        return (_rms(o, 1e-5) * _d(self.norm_w)).reshape(o.shape[0], -1) * gate


# H, G, dk, dv, taps
RULES = [(4, 2, 16, 24, 4), (2, 2, 64, 64, 4), (3, 1, 20, 37, 5), (6, 2, 8, 5, 1), (1, 1, 200, 33, 7), (2, 1, 96, 176, 4), (2, 2, 128, 128, 3),
         (1, 1, 256, 300, 2), (2, 1, 160, 16, 4), (1, 1, 224, 9, 4), (3, 3, 33, 70, 6)]


@pytest.mark.parametrize("H,G,dk,dv,taps", RULES)
def test_delta_rule_whole_in_portions_and_token_by_token(H, G, dk, dv, taps):
    """Three sequences of unequal lengths in one step; the same in portions that start and end anywhere in the records of
    four tokens, mixed with single tokens; one by one; and what each leaves as its state."""
    lens = [41, 3, 70]
    ref = None
    for cuts in ([[41], [3], [70]], [[1, 2, 5, 4, 29], [2, 1], [7, 1, 1, 3, 58]], [[40, 1], [1, 1, 1], [64, 2, 4]]):
        case = Delta(H, G, dk, dv, taps, lens, seed=7)
        ref = ref or [case.reference(i) for i in range(3)]
        at, got = [0, 0, 0], [[], [], []]
        for step in range(max(len(c) for c in cuts)):
            takes = [(i, at[i], cuts[i][step]) for i in (2, 0, 1) if step < len(cuts[i])]
            out, row = case.step(takes), 0
            for i, _, n in takes:
                got[i].append(out[row:row + n])
                row += n
                at[i] += n
        for i in range(3):
            _close(torch.cat(got[i]), ref[i][0], 2e-5)
            _close(case.state[case.slot_of[i]], ref[i][1], 2e-5)
        others = [s for s in range(case.state.shape[0]) if s not in case.slot_of]
        assert float(case.state[others].abs().max()) == 0.0 and float((case.ring[others] - 77.0).abs().max()) == 0.0
    for dtype in (torch.float32, torch.bfloat16):
        case = Delta(H, G, dk, dv, taps, lens, seed=7)
        got = [[], [], []]
        for t in range(max(lens)):
            live = [i for i in (2, 0, 1) if t < lens[i]]
            out = case.single([(i, t) for i in live], dtype)
            for r, i in enumerate(live):
                got[i].append(out[r])
        for i in range(3):
            want = case.finished(i, ref[i][0])
            keep = _firm_heads(ref[i], case).reshape(lens[i], H, 1).expand(-1, -1, dv).reshape(lens[i], -1)
            g = torch.stack(got[i]).double().cpu()
            _close(torch.where(keep, g, want), want, 3e-4 if dtype == torch.float32 else 2 * BF16_ULP, BF16_ULP)
            _close(case.state[case.slot_of[i]], ref[i][1], 2e-5)


def _firm_heads(ref, case):
    """(n, H): heads whose output is not the small rest of a sum that nearly cancels (the norm behind it blows that up)."""
    o = ref[0]
    size = o.pow(2).mean(-1).sqrt()
    return size > 0.03 * size.median()


@pytest.mark.parametrize("dk,dv", [(64, 64), (96, 40), (16, 24)])
def test_a_prompt_goes_on_token_by_token_and_back(dk, dv):
    """A prompt by records, single tokens, a portion, single tokens: both kernels leave each other the same state and the
    same convolution's past."""
    n = 60
    case = Delta(4, 2, dk, dv, 4, [n, n], seed=21)
    ref = [case.reference(i) for i in range(2)]
    raw = case.step([(0, 0, 21), (1, 0, 18)])
    _close(raw[:21], ref[0][0][:21], 2e-5)
    at = [21, 18]
    for k in range(9):
        out = case.single([(1, at[1]), (0, at[0])], torch.float32)
        for r, i in ((0, 1), (1, 0)):
            want = case.finished(i, ref[i][0])[at[i]]
            firm = _firm_heads(ref[i], case)[at[i]].repeat_interleave(dv)
            _close(torch.where(firm, out[r].double().cpu(), want), want, 3e-4)
        at = [p + 1 for p in at]
    raw = case.step([(0, at[0], n - at[0]), (1, at[1], n - at[1])])
    _close(raw[:n - at[0]], ref[0][0][at[0]:], 2e-5)
    _close(raw[n - at[0]:], ref[1][0][at[1]:], 2e-5)


@pytest.mark.parametrize("single", [False, True])
def test_a_write_is_read_back_after_hundreds_of_tokens(single):
    """Nothing decays (rate 0) and only the token at 5 writes (every other step size is sigmoid(-80)): hundreds of tokens
    later a query that equals its key reads its value, and a query at right angles to it reads nothing."""
    n, H, dk, dv = 400, 2, 32, 16
    case = Delta(H, 2, dk, dv, 1, [n], seed=3, rate=0.0)
    rows = case.rows[0]
    rows[:, case.b_off:case.b_off + H] = -80.0
    rows[5, case.b_off:case.b_off + H] = 80.0
    case.taps_w.fill_(1.0)
    rows[:, :2 * 2 * dk] = -30.0                                 # silu of -30 is nothing: every other q and k is small but a unit vector needs one place
    rows[:, 0] = rows[:, dk] = 8.0                               # queries look at channel 0 of either head
    rows[399, 0] = rows[399, dk] = -30.0
    rows[399, 1] = rows[399, dk + 1] = 8.0                       # the last one at channel 1
    rows[:, 2 * dk] = rows[:, 3 * dk] = 8.0                      # keys stand on channel 0
    v5 = rows[5, 4 * dk:4 * dk + H * dv]
    want = (v5 * torch.sigmoid(v5)).reshape(H, dv)
    want = want * dk ** -0.5
    if single:
        out = [case.single([(0, t)], torch.float32)[0] for t in range(n)]
        S = case.state[case.slot_of[0]]
        _close(S[:, 0], want * dk ** 0.5, 1e-5)
        assert float(S[:, 1:].abs().max()) < 1e-6 and torch.isfinite(torch.stack(out)).all()
        return
    out = case.step([(0, 0, n)])
    assert float(out[:5].abs().max()) < 1e-9                     # nothing written yet
    for t in (5, 6, 100, 398):
        _close(out[t], want, 1e-5)
    assert float(out[399].abs().max()) < 1e-4 * float(want.abs().max())
    _close(case.state[case.slot_of[0]][:, 0], want * dk ** 0.5, 1e-5)


@pytest.mark.parametrize("single", [False, True])
def test_decays_of_zero_and_a_slot_that_is_used_again(single):
    """A rate so large that every decay is exactly zero: each position reads its own write alone, in a slot whose ring still
    holds another sequence's rows and whose state starts from zero."""
    case = Delta(3, 1, 24, 40, 4, [30], seed=5, rate=1e6, bias=5.0)
    case.ring.fill_(float("nan"))                                # a former owner's rows: positions below zero are not read
    ref, S = case.reference(0)
    assert torch.isfinite(ref).all()
    if single:
        got = torch.stack([case.single([(0, t)], torch.float32)[0] for t in range(30)])
        want, firm = case.finished(0, ref), _firm_heads((ref, S), case).repeat_interleave(40, dim=1)
        _close(torch.where(firm, got.double().cpu(), want), want, 3e-4)
    else:
        _close(case.step([(0, 0, 30)]), ref, 2e-5)
    _close(case.state[case.slot_of[0]], S, 2e-5)


def test_sizes_that_the_rule_does_not_take_are_refused():
    ops = _ops()
    case = Delta(1, 1, 8, 8, 4, [4], seed=1)
    with pytest.raises(ops.KernelError):
        ops.delta_prompt(case.rows[0], case.b_off, case.taps_w, case.ring[:, :2].contiguous(), case.z(case.rows[0]), case.bias, case.rate, case.state,
                         _i32([0, 4]), _i32([0]), _i32([0, 1, 2, 3]), 1, 4, 1, 1, 8, 8, 1.0, 1e-6)
    with pytest.raises(ops.KernelError):
        ops.attn_prefill(_rand((1, 64), torch.bfloat16, 1), _rand((1, 1, 64, 64), torch.bfloat16, 1), _rand((1, 1, 64, 264), torch.bfloat16, 2),
                         _i32([[0]]), _i32([0]), _i32([1]), _blocks([1], [0], 64), 1, 1, 64, 64, 1.0, None, vd=264)


# ------------------------------------------------------------------ fixed decays through records, gates by pieces

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,dk,dv", [(2, 16, 24), (3, 64, 64), (1, 20, 37), (2, 128, 48), (1, 256, 5), (2, 96, 200), (1, 161, 12)])
def test_fixed_decay_records_whole_in_portions_and_beside_single_tokens(dtype, H, dk, dv):
    """Decays of exactly one, close to one and far from it; whole, in portions, and going on from (and to) the kernel for
    single tokens; a first token that stands out is still there behind a decay of one."""
    ops = _ops()
    lens, decays = [70, 3, 41], [1.0, 0.9995, 0.3][:H]
    decay = torch.tensor(decays, device=DEV)
    off, width = (3, 3 + H * dk, 3 + 2 * H * dk), 3 + 2 * H * dk + H * dv + 2
    rows = [_rand((n, width), dtype, 60 + i) for i, n in enumerate(lens)]
    for r in rows:
        r[0, off[2]:off[2] + H * dv] = 25.0
    ref = []
    for r in rows:
        x = _d(r)
        x = x * torch.sigmoid(x)
        n = x.shape[0]
        q, k = x[:, off[0]:off[0] + H * dk].reshape(n, H, dk), x[:, off[1]:off[1] + H * dk].reshape(n, H, dk)
        v = x[:, off[2]:off[2] + H * dv].reshape(n, H, dv)
        S, o = torch.zeros(H, dk, dv, dtype=torch.float64), torch.zeros(n, H, dv, dtype=torch.float64)
        for t in range(n):
            S = _d(decay)[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
            o[t] = torch.einsum("hdv,hd->hv", S, q[t])
        ref.append((o, S))
    for cuts in ([[70], [3], [41]], [[1, 2, 5, 4, 58], [2, 1], [7, 1, 1, 32]], [[64, -6], [-3], [5, -1, 35]]):       # -n: n single tokens
        state = torch.zeros((5, H, dk, dv), dtype=torch.float32, device=DEV)
        slots, at, got = [4, 0, 2], [0, 0, 0], [[], [], []]
        for i in range(3):
            for c in cuts[i]:
                for n in ([c] if c > 0 else [1] * -c):
                    part = rows[i][at[i]:at[i] + n].contiguous()
                    cu, sl = _i32([0, n]), _i32([slots[i]])
                    if c > 0:
                        out = ops.linear_prompt(part, *off, decay, state, cu, sl, 1, n, H, dk, dv)
                    else:
                        out, _ = ops.linear_scan(part, *off, state, cu, sl, _i32([at[i]]), 1, H, dk, dv, decay=decay, single=True, in_act="silu")
                    got[i].append(out)
                    at[i] += n
        for i in range(3):
            _close(torch.cat(got[i]), ref[i][0], 2e-5)
            _close(state[slots[i]], ref[i][1], 2e-5)
    # all three sequences in one step
    state = torch.zeros((5, H, dk, dv), dtype=torch.float32, device=DEV)
    out = ops.linear_prompt(torch.cat(rows).contiguous(), *off, decay, state, _i32([0, 70, 73, 114]), _i32([4, 0, 2]), 3, 70, H, dk, dv)
    for i, (lo, hi) in enumerate(((0, 70), (70, 73), (73, 114))):
        _close(out[lo:hi], ref[i][0], 2e-5)
    assert float(state[1].abs().max()) == 0.0 and float(state[3].abs().max()) == 0.0


@pytest.mark.parametrize("gdtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("cols,off", [(64, 8), (64, 3), (20, 0), (1024, 16)])
@pytest.mark.parametrize("act", ["sigmoid", "silu"])
def test_gates_by_pieces_and_one_by_one(gdtype, cols, off, act):
    ops = _ops()
    x, wide = _rand((9, cols), torch.bfloat16, 1), _rand((9, cols + 32), gdtype, 2, 3.0)
    gate = wide[:, off:off + cols]
    g = _d(gate)
    ref = _d(x) * (torch.sigmoid(g) if act == "sigmoid" else g * torch.sigmoid(g))
    _close(ops.gate_mul(x.clone(), gate, act), ref, BF16_ULP, BF16_ULP)
