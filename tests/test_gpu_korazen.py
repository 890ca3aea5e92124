"""The Korazen design through the engine: every mechanism alone and together, every way of cutting and batching requests,
slots and pages used again, long decoding, the edges of blocks made visible by one odd token, the first token carried by
the states, generation through the entry point and the command line -- each against the plain implementation
(tests/plain_korazen.py)."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_korazen
from korazen_models import CONFIGS, bound, firm_rows, load, make_folder, random_config, rewrite, row_errors, tokens
from trace_tools import ROOT, Trace, run_trace, split, trace_batches, trace_chunked, trace_last_one_by_one, trace_mixed, trace_whole

pytestmark = pytest.mark.gpu

DTYPES = ["float32", "bfloat16"]


def _engine(folder, dtype, **kw):
    from longbow_quarrel_b200.engine import Engine
    return Engine.from_pretrained(folder, dtype=dtype, **kw)


_memo: dict = {}


def _plain(folder, toks, dtype=None):
    """The plain implementation's logits for a request and, with a dtype, its bound and firm rows (kept: every cut is compared
    with them)."""
    key = (str(folder), tuple(toks))
    if key not in _memo:
        cfg, weights = load(folder)
        margins: list = []
        _memo[key] = {"ref": plain_korazen.forward(cfg, weights, toks, margins=margins).numpy(), "margins": margins}
    entry = _memo[key]
    if dtype is not None and dtype not in entry:
        firm = firm_rows(dtype, *load(folder), toks, entry["margins"])
        entry[dtype] = (bound(dtype, *load(folder), toks, entry["ref"], firm), firm)
    return entry["ref"] if dtype is None else (entry["ref"], *entry[dtype])


def _check(got: dict, requests: dict, folder, dtype: str, what: str):
    """float32: every row within its request's bound.  bfloat16: no row beyond one and a half times the bound and at
    most one row in fifty beyond the bound itself."""
    over = total = 0
    for rid, toks in requests.items():
        ref, tol, firm = _plain(folder, toks, dtype)
        keys = [k for k in got if k[0] == rid]
        assert keys, f"{what}: nothing came back for {rid}"
        for _, pos in keys:
            if not firm[pos]:
                continue
            err = float(row_errors(got[(rid, pos)], ref[pos]))
            hard = tol if dtype == "float32" else 1.5 * tol
            assert err < hard, f"{what}: request {rid} position {pos} of {len(toks)}: error {err:.3g}, bound {hard:.3g}"
            over += err >= tol
            total += 1
    assert total > 0 and over <= 0.02 * total, f"{what}: {over} of {total} rows over their bound"


def _rows(eng, slot, toks, cut):
    """The logits of every position: the first `cut` tokens in one step, the others one by one."""
    rows = [eng.step([(slot, toks[:cut])], [list(range(cut))]).cpu().numpy()] if cut else []
    rows += [eng.step([(slot, [t])], [[0]]).cpu().numpy() for t in toks[cut:]]
    return np.concatenate(rows)


# ------------------------------------------------------------------ each mechanism alone

ALONE = [name for name in sorted(CONFIGS) if name.startswith("only_")]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ALONE)
def test_one_layer_of_each_kind_whole_and_token_by_token(tmp_path, name, dtype):
    """A model of one mechanism: the whole prompt in one step (its first tokens included), and the same tokens one by one
    from the first (133 steps: across two page borders and past most blocks; replayed from a captured step)."""
    folder = make_folder(tmp_path, name, seed=3, keep_ranks=False)
    toks = tokens(133, CONFIGS[name]["vocab"], 5)
    ref, tol, firm = _plain(folder, toks, dtype)
    assert firm.sum() > 60
    eng = _engine(folder, dtype, max_tokens=512)
    s = eng.new_sequence()
    whole = _rows(eng, s, toks, len(toks))
    eng.end_sequence(s)
    assert row_errors(whole, ref)[firm].max() < tol
    s = eng.new_sequence()
    single = _rows(eng, s, toks, 0)
    eng.end_sequence(s)
    assert row_errors(single, ref)[firm].max() < tol
    assert row_errors(single, whole)[firm].max() < tol
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["only_delta", "only_sides"])
def test_a_checkpoint_stored_in_32_bit(tmp_path, name, dtype):
    """Every tensor float32: the products keep them as they are, in either precision of the model."""
    folder = make_folder(tmp_path, name, seed=6, dtype=torch.float32)
    toks = tokens(70, CONFIGS[name]["vocab"], 9)
    ref, tol, firm = _plain(folder, toks, dtype)
    import warnings
    with warnings.catch_warnings():
        warnings.simplefilter("ignore")                      # (the loader says that such products run on the CUDA cores)
        eng = _engine(folder, dtype, max_tokens=256)
    s = eng.new_sequence()
    assert row_errors(_rows(eng, s, toks, 40), ref)[firm].max() < tol
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_block_ends_where_it_ends_when_one_token_outweighs_all_others(tmp_path, dtype):
    """The softmax side alone (the other side's norm weight is zero), in a prompt of one odd token among copies of another
    and with a flat softmax, so that one odd key shows.  With blocks of 4 an odd token at position 30 changes the logits
    of 30 and 31 and none from 32 on, one at 31 its own row alone, one at 28 (the block's first) the whole block; with
    blocks of 64 one at 63 its own row alone (a page's last place) and one at 64 the rows up to 127 -- in a prompt, with
    the edge among decoded tokens, and with everything after the odd token decoded."""
    for size, cases in ((4, [(30, 31), (31, 31), (28, 31)]), (64, [(63, 63), (64, 127)])):
        data = json.loads(json.dumps(CONFIGS["only_sides_wide_values"]))
        data["layers"][0]["mixer"]["left"].update(mask={"size": size}, scale=0.02)
        folder = make_folder(tmp_path / str(size), data, seed=9, std=0.5)
        rewrite(folder, lambda w: w["l0.mix.right.out"].zero_())
        n = 70 if size == 4 else 135
        base = [7] * n
        ref_base = _plain(folder, base)
        eng = _engine(folder, dtype, max_tokens=512)
        for at, inside in cases:
            outside = inside + 1
            odd = list(base)
            odd[at] = 55
            ref_odd, tol, _ = _plain(folder, odd, dtype)
            assert row_errors(ref_odd[inside], ref_base[inside]) > 1e-3
            assert row_errors(ref_odd[outside:], ref_base[outside:]).max() < 1e-12
            for cut in (n, max(at + 1, inside - 3), at + 1):
                s = eng.new_sequence()
                got = _rows(eng, s, odd, cut)
                eng.end_sequence(s)
                assert row_errors(got, ref_odd).max() < tol, (size, at, cut)
                # (an odd key among sixty-four weighs about what rounding to bfloat16 does: the float32 run shows it)
                if size == 4 or inside == at or dtype == "float32":
                    assert row_errors(got[inside], ref_base[inside]) > 2 * tol, (size, at, cut)
                assert row_errors(got[outside:], ref_base[outside:]).max() < tol, (size, at, cut)
        eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["only_delta", "only_delta_even", "only_sides_open"])
def test_the_first_token_lasts_in_the_states(tmp_path, name, dtype):
    """Decays so close to one that the first of 300 tokens still shows at the last: in the delta rule's state (with small
    step sizes, so that later writes leave it standing) and in the fixed-decay state, whole, with the last 200 decoded and
    in portions that end off the record's four tokens."""
    data = json.loads(json.dumps(CONFIGS[name]))
    if name == "only_sides_open":
        data["layers"][0]["mixer"]["right"]["decay"] = [0.9999, 1.0]
    folder = make_folder(tmp_path, data, seed=4, std=0.5)

    def change(w):
        if name == "only_sides_open":
            w["l0.mix.left.out"].zero_()
        else:
            w["l0.mix.dt_bias"].fill_(-14.0)
            w["l0.mix.a2"].mul_(0.01)
            w["l0.mix.b"].mul_(0.1)
    rewrite(folder, change)
    base = tokens(300, data["vocab"], 8)
    odd = [(base[0] + 1) % data["vocab"]] + base[1:]
    ref_base, (ref_odd, tol, firm) = _plain(folder, base), _plain(folder, odd, dtype)
    sharp = row_errors(ref_odd[299], ref_base[299]) > 5 * tol
    assert sharp or dtype == "bfloat16"                      # one token among three hundred may be as small as rounding to bfloat16
    eng = _engine(folder, dtype, max_tokens=512)
    for portions in ([300], [100] + [1] * 200, [97, 2, 3, 1, 101, 96]):
        s = eng.new_sequence()
        rows, at = [], 0
        for n in portions:
            rows.append(eng.step([(s, odd[at:at + n])], [list(range(n))]).cpu().numpy())
            at += n
        eng.end_sequence(s)
        got = np.concatenate(rows)
        assert row_errors(got, ref_odd)[firm].max() < tol, portions[:3]
        assert not sharp or row_errors(got[299], ref_base[299]) > 3 * tol, portions[:3]
    eng.close()


# ------------------------------------------------------------------ whole models, every cut, through the replay program

LENGTHS = {"r0": 70, "r1": 33, "r2": 140, "r3": 65, "r4": 64, "r5": 34, "r6": 129}
PROMPTS = {"r0": 7, "r1": 1, "r2": 100, "r3": 2, "r4": 63, "r5": 20, "r6": 65}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
def test_every_cut_of_every_request_matches_plain(tmp_path, name, dtype):
    """Whole; the last 32 tokens one by one; batches of three unequal requests that go on together, the shorter
    ending earlier, the next batch in the slots and pages given back; portions of 2, 3, 59, 1, 64 and 7 tokens;
    steps that mix portions with single tokens.  One call of the replay program runs them one after the other."""
    folder = make_folder(tmp_path, name, seed=11, keep_ranks=False)
    vocab = CONFIGS[name]["vocab"]
    requests = {rid: tokens(n, vocab, 100 + i) for i, (rid, n) in enumerate(LENGTHS.items())}
    tr = Trace()
    tr.extend(trace_whole(requests), "whole:")
    tr.extend(trace_last_one_by_one(requests), "tail:")
    tr.extend(trace_batches(requests, PROMPTS, width=3), "batched:")
    tr.extend(trace_chunked(requests, [2, 3, 59, 1, 64, 7]), "portions:")
    tr.extend(trace_mixed(requests, PROMPTS, [5, 1, 2, 1, 17]), "mixed:")
    got = run_trace(folder, dtype, tr, tmp_path / "out")
    cuts = {p: split(got, p + ":") for p in ("whole", "tail", "batched", "portions", "mixed")}
    for what, rows in cuts.items():
        assert len(rows) == (33 * len(requests) if what == "tail" else sum(LENGTHS.values())), what
        _check(rows, requests, folder, dtype, what)
    if dtype == "float32":
        for rid, toks in requests.items():
            _, tol, firm = _plain(folder, toks, dtype)
            for what in ("tail", "batched", "portions", "mixed"):
                for (r, pos), row in cuts[what].items():
                    if r == rid and firm[pos]:
                        err = float(row_errors(row, cuts["whole"][(r, pos)]))
                        assert err < 2 * tol, f"{what} against whole: {rid} position {pos}: {err:.3g}, bound {2 * tol:.3g}"


@pytest.mark.parametrize("seed", [3, 12])
def test_configurations_drawn_at_random_match_plain(tmp_path, seed):
    """Sizes and options that nobody chose: whole, the last 30 tokens one by one and an unequal batch, in both precisions."""
    import random
    rng = random.Random(seed)
    folder = make_folder(tmp_path, random_config(rng), seed=seed, std=rng.choice([0.1, 0.2]))
    cfg, _ = load(folder)
    requests = {rid: tokens(n, cfg["vocab"], 50 * seed + i) for i, (rid, n) in enumerate({"a": 150, "b": 70, "c": 33}.items())}
    tr = Trace()
    tr.extend(trace_whole(requests), "whole:")
    tr.extend(trace_last_one_by_one(requests, n_last=30), "tail:")
    tr.extend(trace_batches(requests, {"a": 110, "b": 40, "c": 3}, width=3), "batched:")
    for dtype in DTYPES:
        got = run_trace(folder, dtype, tr, tmp_path / ("out_" + dtype))
        for what in ("whole", "tail", "batched"):
            _check(split(got, what + ":"), requests, folder, dtype, f"seed {seed} {dtype} {what}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_stream_after_every_layer_matches_plain(tmp_path, dtype):
    """The residual stream after each layer, for a prompt that is longer than every block, and for the same in portions."""
    folder = make_folder(tmp_path, "mixed", seed=13)
    toks = tokens(150, CONFIGS["mixed"]["vocab"], 17)
    cfg, weights = load(folder)
    exact: list = []
    plain_korazen.forward(cfg, weights, toks, layers_out=exact)
    other: list = []
    kw = {"dtype": torch.float32} if dtype == "float32" else {"storage": torch.bfloat16}
    plain_korazen.forward(cfg, weights, toks, layers_out=other, **kw)
    firm = firm_rows(dtype, cfg, weights, toks)
    eng = _engine(folder, dtype, max_tokens=512)
    for portions in ([150], [64, 1, 2, 83]):
        seen: dict = {}
        eng.model.probe = lambda i, x, ctx: seen.setdefault(i, []).append(x.detach().float().cpu().clone())
        s = eng.new_sequence()
        at = 0
        for n in portions:
            eng.step([(s, toks[at:at + n])], [[n - 1]])
            at += n
        eng.end_sequence(s)
        eng.model.probe = None
        for i in range(5):
            got = torch.cat(seen[i]).numpy()
            yard = max(1e-5, 3.0 * float(row_errors(other[i].numpy(), exact[i].numpy())[firm].max()))
            assert row_errors(got, exact[i].numpy())[firm].max() < yard, (portions, i)
    eng.close()


# ------------------------------------------------------------------ slots and pages used again, long decoding

@pytest.mark.parametrize("dtype", DTYPES)
def test_a_slot_that_is_used_again_starts_from_nothing(tmp_path, dtype):
    """One slot and just enough pages: each request runs in what the one before it gave back, so a state, a convolution's
    last inputs or a page that outlived its request would show in the next one's first tokens."""
    folder = make_folder(tmp_path, "mixed", seed=21)
    eng = _engine(folder, dtype, max_tokens=192, max_batch=1)
    rows, requests = {}, {}
    for i, n in enumerate([150, 3, 130, 66]):
        toks = requests[i] = tokens(n, CONFIGS["mixed"]["vocab"], 300 + i)
        s = eng.new_sequence()
        assert s == 0
        got = _rows(eng, s, toks, max(1, n - 40))
        eng.end_sequence(s)
        rows.update({(i, p): row for p, row in enumerate(got)})
    _check(rows, requests, folder, dtype, "one slot")
    assert eng.cache.pages_in_use() == 0
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_from_the_first_token(tmp_path, dtype):
    """260 single-token steps of three sequences side by side (captured once, replayed): the blocks of 64 and 100 pass wholly
    over decoded tokens, their pages go back and come to other sequences, and the states are carried over hundreds of steps."""
    folder = make_folder(tmp_path, "mixed", seed=31)
    vocab = CONFIGS["mixed"]["vocab"]
    seqs = [tokens(260, vocab, 40), tokens(260, vocab, 41), tokens(150, vocab, 42)]
    eng = _engine(folder, dtype, max_tokens=3 * 320)
    slots = [eng.new_sequence() for _ in seqs]
    got = {}
    for t in range(260):
        live = [i for i, q in enumerate(seqs) if t < len(q)]
        out = eng.step([(slots[i], [seqs[i][t]]) for i in live], [[0]] * len(live)).cpu().numpy()
        for row, i in zip(out, live):
            got[(i, t)] = row
            if t == len(seqs[i]) - 1:
                eng.end_sequence(slots[i])
    _check(got, dict(enumerate(seqs)), folder, dtype, "decoded")
    eng.close()


# ------------------------------------------------------------------ generation through the entry point and the command line

def _greedy_matches(folder, prompt, new, dtype):
    cfg, weights = load(folder)
    seq = list(prompt)
    for tok in new:
        margins: list = []
        logits = plain_korazen.forward(cfg, weights, seq, margins=margins)[-1].numpy()
        best = int(np.argmax(logits))
        gap = (logits[best] - logits[tok]) / np.sqrt((logits ** 2).mean())
        if not firm_rows(dtype, cfg, weights, seq, margins)[-1]:
            seq.append(tok)                                  # a read-out that nearly cancels: go on from what was generated
            continue
        assert tok == best or (dtype == "bfloat16" and gap < 5e-2), (dtype, len(seq), tok, best, gap)
        seq.append(tok)


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_scheduler(tmp_path, dtype):
    """Engine.generate: unequal prompts in batches of three (the second batch in the first one's slots), greedy."""
    from longbow_quarrel_b200.sampling import SamplingParams
    folder = make_folder(tmp_path, "mixed", seed=41)
    vocab = CONFIGS["mixed"]["vocab"]
    prompts = [tokens(n, vocab, 500 + i) for i, n in enumerate([9, 1, 70, 2, 64])]
    eng = _engine(folder, dtype, max_tokens=3 * 128, max_batch=3)
    out = eng.generate(prompts, max_new_tokens=10, sampling=SamplingParams(temperature=0.0), stop_ids=[], batch_size=3)
    assert [len(o) for o in out] == [10] * 5
    for prompt, new in zip(prompts, out):
        _greedy_matches(folder, prompt, new, dtype)
    eng.close()


def test_the_command_line_generates_with_a_korazen_folder(tmp_path):
    folder = make_folder(tmp_path, "odd", seed=51, keep_ranks=False)
    prompt = tokens(12, CONFIGS["odd"]["vocab"], 7)
    proc = subprocess.run([str(ROOT / "bin" / "quarrel"), "-model", str(folder), "-prompt-ids", ",".join(map(str, prompt)),
                           "-n", "6", "-temp", "0", "-penalty", "1.0", "-dtype", "float32", "-output", "json"],
                          capture_output=True, text=True, timeout=600, env={**os.environ, "LQ_PYTHON": sys.executable})
    assert proc.returncode == 0, proc.stderr[-3000:]
    new = json.loads(proc.stdout.strip().splitlines()[-1])["output"][0]
    assert len(new) == 6
    _greedy_matches(folder, prompt, new, "float32")


def test_random_weights_from_a_configuration_and_the_kernels_that_served_it():
    """Engine.from_config builds the design from a dict with config.json's keys; in bfloat16 a prompt of seven hundred
    tokens and decoded tokens go through the design's kernels: the delta rule's records and scan for the prompt and its
    one kernel for single tokens, attention on the tensor cores (also where values have a size of their own), the
    fixed-decay scan in both forms, both forms of the kernel in which branches join the stream."""
    from longbow_quarrel_b200.engine import Engine
    from longbow_quarrel_b200.kernels import ops
    from longbow_quarrel_b200.sampling import SamplingParams
    eng = Engine.from_config(CONFIGS["wide"], seed=3, max_tokens=2048, max_batch=2)
    before = ops.launches_by_name()
    out = eng.generate([[t % 300 for t in range(1, 701)], [4]], max_new_tokens=5, sampling=SamplingParams(temperature=0.0), stop_ids=[])
    ran = ops.launches_since(before)
    assert [len(o) for o in out] == [5, 5]
    for kernel in ("embedding_norm", "delta_prompt", "delta_single", "join_normed", "join_normed:two", "rope_partial", "attn_prefill_tc",
                   "attn_prefill:vd", "attn_decode:teams", "linear_scan", "linear_scan:single", "head_norm_gate", "gate_mul"):
        assert ran.get(kernel, 0) >= 1, (kernel, ran)
    for kernel in ("attention", "gated_act", "swiglu", "add_bias"):     # the plain attention served no layer; nothing fused ran apart
        assert ran.get(kernel, 0) == 0, (kernel, ran)
    eng.close()
