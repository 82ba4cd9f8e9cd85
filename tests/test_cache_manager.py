"""The page pool and the cache manager on the CPU: no page lost, held twice or freed twice, under random
orders of requests; windowed release; fixed-size state slots."""
import random

import pytest
import torch

from flambeau_b200.cache.manager import CacheManager, CallPlan
from flambeau_b200.cache.pages import Books, OutOfPages, PageError
from flambeau_b200.parts.base import KVRequirement, StateRequirement


class PagePool:
    """A pool on its own, driven through the books (one group, one request slot per held page, pages of one
    token): what the cache manager's groups are made of."""

    def __init__(self, n_pages: int):
        if n_pages <= 0:
            raise ValueError("a page pool needs at least one page")
        self.n_pages = int(n_pages)
        # one request slot per possible holder of a single page; page_size 1 makes a token a page
        self._books = Books([self.n_pages], [0], 1, self.n_pages + 1, self.n_pages)
        self._holder: dict = {}              # page id -> slot that holds it

    @property
    def n_free(self) -> int:
        return self._books.free_pages()[0]

    @property
    def n_held(self) -> int:
        return self.n_pages - self.n_free

    def take(self, count: int) -> list:
        """`count` page ids, or OutOfPages with nothing taken."""
        if count < 0:
            raise ValueError("negative page count")
        if count > self.n_free:
            raise OutOfPages(count, self.n_free, self.n_pages)
        out = []
        for _ in range(count):
            slot = self._books.admit()
            self._books.reserve_all([slot], [1])
            page = self._books.pages(slot, 0)[0]
            self._holder[page] = slot
            out.append(page)
        return out

    def give_back(self, pages) -> None:
        for p in pages:
            if not 0 <= p < self.n_pages:
                raise PageError(f"page id {p} is outside the pool of {self.n_pages}")
            slot = self._holder.pop(p, None)
            if slot is None:
                raise PageError(f"page {p} is given back but is not held")
            self._books.release(slot)

    def is_held(self, page: int) -> bool:
        return self._books.is_held(0, page)


def test_pool_is_fifo_and_all_or_nothing():
    pool = PagePool(4)
    a = pool.take(3)
    assert a == [0, 1, 2] and pool.n_free == 1
    with pytest.raises(OutOfPages):
        pool.take(2)
    assert pool.n_free == 1                      # nothing was taken
    pool.give_back([1])
    assert pool.take(2) == [3, 1]                # reused in the order of return
    with pytest.raises(PageError):
        pool.give_back([0, 0])                   # freed twice
    with pytest.raises(PageError):
        pool.give_back([7])


def manager(window=0, tokens=256, layers=2, max_requests=4, state=False, max_seq_len=None):
    plans = [CallPlan(kv=KVRequirement(2, 16, window), state=StateRequirement((3,)) if state else None)
             for _ in range(layers)]
    return CacheManager(plans, max_tokens=tokens, page_size=16, max_requests=max_requests, device="cpu",
                        dtype=torch.float32, max_seq_len=max_seq_len or tokens)


def test_groups_follow_requirements():
    plans = [CallPlan(kv=KVRequirement(2, 16, 0)), CallPlan(kv=KVRequirement(2, 16, 8)),
             CallPlan(kv=KVRequirement(2, 16, 0)), CallPlan(kv=None, state=StateRequirement((5,))),
             CallPlan(kv=KVRequirement(2, 16, 0), cache_from=0)]
    cm = CacheManager(plans, max_tokens=64, page_size=16, max_requests=2, device="cpu", dtype=torch.float32)
    assert cm.n_groups == 2
    assert cm.group_of_call[0] == cm.group_of_call[2] == cm.group_of_call[4] != cm.group_of_call[1]
    assert 3 not in cm.group_of_call and cm.state[3].shape == (2, 5)
    v = cm.view(4, [None, None])
    assert not v.writable and v.k_pool is cm.groups[cm.group_of_call[0]].k[0]
    assert cm.view(2, [None, None]).writable
    with pytest.raises(ValueError):
        CacheManager([CallPlan(kv=None), CallPlan(kv=KVRequirement(1, 8), cache_from=0)], max_tokens=64,
                     page_size=16, max_requests=1, device="cpu", dtype=torch.float32)


def test_reserve_is_all_or_nothing_and_release_returns_everything():
    cm = manager(tokens=64)                      # 4 pages
    cm.admit("a")
    cm.reserve("a", 40)                          # 3 pages
    cm.commit("a", 40)
    cm.admit("b")
    assert not cm.can_reserve([("b", 17)])
    with pytest.raises(OutOfPages):
        cm.reserve("b", 17)
    assert cm.free_pages() == [1]
    cm.reserve("b", 16)
    cm.commit("b", 16)
    cm.check_invariants()
    cm.release("a")
    cm.release("b")
    assert cm.free_pages() == [4] and not cm.requests
    with pytest.raises(KeyError):
        cm.release("a")


def test_window_gives_pages_back_as_they_die():
    cm = manager(window=16, tokens=64, max_seq_len=128)
    cm.admit("a")
    held = []
    for _ in range(10):                          # 100 tokens through a 4-page pool
        cm.reserve("a", 10)
        cm.commit("a", 10)
        cm.check_invariants()
        held.append(4 - cm.free_pages()[0])
    assert max(held) <= 3
    rec = cm.requests["a"]
    first_live = rec.length - 16 + 1
    for j, p in enumerate(rec.pages[0]):
        assert (p < 0) == ((j + 1) * 16 <= first_live), "exactly the pages wholly below the window are given back"
    assert cm.first_live_page("a", 0) == first_live // 16
    cm.release("a")
    assert cm.free_pages() == [4]


def test_commit_beyond_reservation_is_an_error():
    cm = manager()
    cm.admit("a")
    cm.reserve("a", 5)
    with pytest.raises(PageError):
        cm.commit("a", 6)


def test_state_slots_are_zeroed_on_admission_and_reused():
    cm = manager(state=True, max_requests=2)
    a = cm.admit("a")
    cm.state[0][a.slot] += 5.0
    b = cm.admit("b")
    assert a.slot != b.slot
    with pytest.raises(PageError):
        cm.admit("c")
    cm.release("a")
    c = cm.admit("c")
    assert c.slot == a.slot and float(cm.state[0][c.slot].abs().sum()) == 0.0
    assert cm.state_bytes_per_request() == 2 * 3 * 4


@pytest.mark.parametrize("window", [0, 16, 40])
@pytest.mark.parametrize("seed", range(5))
def test_random_orders_never_lose_or_double_a_page(window, seed):
    rng = random.Random(seed)
    cm = manager(window=window, tokens=192, max_requests=4)
    live, next_id = {}, 0
    for _ in range(400):
        r = rng.random()
        if r < 0.25 and cm.has_slot():
            cm.admit(next_id)
            live[next_id] = 0
            next_id += 1
        elif r < 0.85 and live:
            rid = rng.choice(list(live))
            k = rng.choice([1, 1, 1, 2, 5, 17, 33])
            if cm.can_reserve([(rid, k)]) and cm.length(rid) + k <= 192:
                before = cm.free_pages()
                cm.reserve(rid, k)
                cm.commit(rid, k)
                live[rid] += k
                assert cm.length(rid) == live[rid]
                if window == 0:
                    assert before[0] - cm.free_pages()[0] == -(-live[rid] // 16) - -(-(live[rid] - k) // 16)
            else:
                free = cm.free_pages()
                if not cm.can_reserve([(rid, k)]):
                    with pytest.raises(OutOfPages):
                        cm.reserve(rid, k)
                    assert cm.free_pages() == free
        elif live:
            rid = rng.choice(list(live))
            cm.release(rid)
            del live[rid]
        cm.check_invariants()
        held = sum(sum(1 for p in rec.pages[0] if p >= 0) for rec in cm.requests.values())
        assert held + cm.free_pages()[0] == cm.groups[0].pool.n_pages
    cm.release_all()
    assert cm.free_pages() == [12]


def test_a_reader_may_not_look_further_back_than_the_cache_it_reads_keeps():
    """Pages are given back by the owner's window; a call that reads that cache with no window, or a wider one,
    would ask for keys whose pages are gone."""
    def build(owner_window, reader_window):
        return CacheManager([CallPlan(kv=KVRequirement(2, 16, owner_window)),
                             CallPlan(kv=KVRequirement(2, 16, reader_window), cache_from=0)],
                            max_tokens=64, page_size=16, max_requests=1, device="cpu", dtype=torch.float32)
    for owner, reader in ((16, 0), (16, 32)):
        with pytest.raises(ValueError, match="keeps only"):
            build(owner, reader)
    for owner, reader in ((0, 0), (0, 8), (32, 32), (32, 8)):
        build(owner, reader)


def test_a_windowed_request_outlives_its_table_row():
    """A block-table row holds live pages only, so a request under a window runs on far past the number of
    tokens that the row's columns could address from position 0."""
    plans = [CallPlan(kv=KVRequirement(1, 8, 24))]
    cm = CacheManager(plans, max_tokens=128, page_size=8, max_requests=2, device="cpu", dtype=torch.float32,
                      max_seq_len=100000, max_step_tokens=16)
    assert cm.table_pages == -(-(24 + 16) // 8) + 2
    cm.admit("a")
    for _ in range(300):                          # 4,800 tokens through a row of 7 columns and a pool of 16 pages
        cm.reserve("a", 16)
        live = [p for p in cm.requests["a"].pages[0] if p >= 0]
        assert len(live) <= cm.table_pages
        cm.commit("a", 16)
        cm.check_invariants()
    assert cm.length("a") == 4800 and cm.first_live_page("a", 0) == (4800 - 24 + 1) // 8


@pytest.mark.parametrize("window", [0, 24])
def test_snapshot_and_restore_bring_a_request_back(window):
    """What a request holds goes to the host and comes back into other pages and another slot: same length, same
    first live page, same contents by logical page, same state; all or nothing when pages are short."""
    plans = [CallPlan(kv=KVRequirement(2, 4, window), state=StateRequirement((3,))), CallPlan(kv=KVRequirement(2, 4, window))]
    cm = CacheManager(plans, max_tokens=128, page_size=8, max_requests=4, device="cpu", dtype=torch.float32,
                      max_seq_len=512)
    g = cm.groups[0]
    for t in list(g.k.values()) + list(g.v.values()):
        t.copy_(torch.arange(t.numel(), dtype=torch.float32).view_as(t))     # every element names its place
    cm.admit("a")
    for _ in range(9):
        cm.reserve("a", 7)
        cm.commit("a", 7)                                                      # 63 tokens; under the window pages go back
    cm.state[0][cm.requests["a"].slot] = torch.tensor([1.0, 2.0, 3.0])
    before_pages = [p for p in cm.requests["a"].pages[0]]
    live = [p for p in before_pages if p >= 0]
    snap = cm.snapshot("a")
    assert snap.length == 63 and snap.first_pages == [cm.first_live_page("a", 0)]
    assert snap.k[0].shape[0] == len(live) and torch.equal(snap.k[1], g.k[1][live])
    cm.release("a")
    cm.admit("other")
    cm.reserve("other", 20)                                                    # takes the pages that came back first
    cm.commit("other", 20)
    for t in list(g.k.values()) + list(g.v.values()):
        t.zero_()
    cm.restore("b", snap)
    cm.check_invariants()
    rec = cm.requests["b"]
    assert rec.length == 63 and cm.first_live_page("b", 0) == snap.first_pages[0]
    after = [p for p in rec.pages[0]]
    assert [p < 0 for p in after] == [p < 0 for p in before_pages]
    now_live = [p for p in after if p >= 0]
    assert now_live != live, "the request came back into other pages"
    for c in (0, 1):
        assert torch.equal(g.k[c][now_live], snap.k[c]) and torch.equal(g.v[c][now_live], snap.v[c])
    assert cm.state[0][rec.slot].tolist() == [1.0, 2.0, 3.0]
    cm.reserve("b", 5)                                                         # and goes on
    cm.commit("b", 5)
    assert cm.length("b") == 68
    with pytest.raises(PageError):
        cm.restore("b", snap)                                                  # already live
    free = cm.free_pages()
    big = cm.snapshot("b")
    cm.admit("hog")
    cm.reserve("hog", free[0] * 8)
    with pytest.raises(OutOfPages):
        cm.restore("c", big)
    assert cm.free_pages() == [0] and "c" not in cm.requests
    cm.check_invariants()


@pytest.mark.parametrize("keep_first", [1, 8, 9, 30])
def test_a_window_gives_back_all_but_the_pages_of_the_kept_first_keys(keep_first):
    """Under a window that keeps a request's first keys visible, the pages that hold those keys stay while the request
    lives; everything between them and the window goes back as it dies.  A table row is the kept pages, then the live
    ones, and a request runs on far past what the row could address from position 0."""
    page, window = 8, 24
    kept = -(-keep_first // page)
    req = KVRequirement(1, 8, window, keep_first=keep_first)
    assert req.kept_pages(page) == kept and KVRequirement(1, 8, 0, keep_first=keep_first).kept_pages(page) == 0
    cm = CacheManager([CallPlan(kv=req)], max_tokens=160, page_size=page, max_requests=2, device="cpu",
                      dtype=torch.float32, max_seq_len=100000, max_step_tokens=16)
    assert cm.table_pages == -(-(window + 16) // page) + 2 + kept
    cm.admit("a")
    for _ in range(200):
        cm.reserve("a", 16)
        live = [p for p in cm.requests["a"].pages[0] if p >= 0]
        assert len(live) <= cm.table_pages
        cm.commit("a", 16)
        cm.check_invariants()
    length = cm.length("a")
    first_live = length - window + 1
    pages = list(cm.requests["a"].pages[0])
    for j, p in enumerate(pages):
        assert (p < 0) == (j >= kept and (j + 1) * page <= first_live), j
    assert cm.first_live_page("a", 0) == first_live // page
    held = sum(1 for p in pages if p >= 0)
    assert held == kept + len(pages) - first_live // page
    assert cm.free_pages() == [20 - held]
    # a second request takes what the first gave back, and both leave everything behind
    cm.admit("b")
    cm.reserve("b", 5)
    cm.commit("b", 5)
    assert list(cm.requests["b"].pages[0]) and cm.first_live_page("b", 0) == kept, "nothing given back yet"
    cm.release("a")
    cm.release("b")
    assert cm.free_pages() == [20]


def test_the_step_descriptor_lists_kept_pages_in_front_of_the_live_ones():
    from flambeau_b200.engine.batch import BatchBuffers, Entry
    page = 4
    plans = [CallPlan(kv=KVRequirement(1, 8, 6, keep_first=5)), CallPlan(kv=KVRequirement(1, 8, 6))]
    cm = CacheManager(plans, max_tokens=64, page_size=page, max_requests=2, device="cpu", dtype=torch.float32,
                      max_seq_len=1000, max_step_tokens=8)
    buffers = BatchBuffers(torch.device("cpu"), 8, 2, cm.n_groups, cm.table_pages)
    cm.admit("a")
    cm.reserve("a", 3)
    batch = buffers.build([Entry("a", [1, 2, 3], [])], cm, 100)
    kept_group = cm.group_of_call[0]
    row = buffers.h_tables[kept_group, 0].tolist()
    logical = list(cm.requests["a"].pages[kept_group])
    assert row[:2] == [logical[0], -1] and all(p == -1 for p in row[2:]), "two columns for the kept pages, one filled"
    cm.commit("a", 3)
    for _ in range(6):
        cm.reserve("a", 5)
        cm.commit("a", 5)                                         # 33 tokens: the window has passed pages 2 to 5
    cm.reserve("a", 2)
    batch = buffers.build([Entry("a", [1, 2], [1])], cm, 100)
    logical = list(cm.requests["a"].pages[kept_group])
    base = cm.first_live_page("a", kept_group)
    assert base == (33 - 6 + 1) // page and logical[2:base] == [-1] * (base - 2)
    row = buffers.h_tables[kept_group, 0].tolist()
    assert row[:2] == logical[:2] and row[2:2 + len(logical) - base] == logical[base:]
    assert int(buffers.h_seqs[4 + kept_group, 0]) == base
    other = cm.group_of_call[1]
    assert buffers.h_tables[other, 0].tolist()[:len(logical) - base] == list(cm.requests["a"].pages[other])[base:]
    assert batch.n_tokens == 2


def test_snapshot_and_restore_keep_the_kept_pages():
    plans = [CallPlan(kv=KVRequirement(2, 4, 24, keep_first=10))]
    cm = CacheManager(plans, max_tokens=160, page_size=8, max_requests=4, device="cpu", dtype=torch.float32,
                      max_seq_len=512)
    g = cm.groups[0]
    for t in list(g.k.values()) + list(g.v.values()):
        t.copy_(torch.arange(t.numel(), dtype=torch.float32).view_as(t))
    cm.admit("a")
    for _ in range(11):
        cm.reserve("a", 7)
        cm.commit("a", 7)                                                      # 77 tokens
    before = list(cm.requests["a"].pages[0])
    live = [p for p in before if p >= 0]
    assert [p >= 0 for p in before[:2]] == [True, True] and before[2] == -1
    snap = cm.snapshot("a")
    assert snap.k[0].shape[0] == len(live) and torch.equal(snap.k[0], g.k[0][live])
    cm.release("a")
    cm.admit("other")
    cm.reserve("other", 30)
    cm.commit("other", 30)
    cm.restore("b", snap)
    cm.check_invariants()
    after = list(cm.requests["b"].pages[0])
    assert [p < 0 for p in after] == [p < 0 for p in before] and cm.length("b") == 77
    now_live = [p for p in after if p >= 0]
    assert torch.equal(g.k[0][now_live], snap.k[0]) and torch.equal(g.v[0][now_live], snap.v[0])
    cm.reserve("b", 40)
    cm.commit("b", 40)
    assert all(p >= 0 for p in list(cm.requests["b"].pages[0])[:2]), "the kept pages are still there"
    cm.release_all()
    assert cm.free_pages() == [20]


@pytest.mark.parametrize("chunk", [1, 5, 8, 20, 24, 64])
def test_a_chunk_is_given_back_when_the_request_leaves_it(chunk):
    """A query sees its own chunk of positions only: once the next position lies in another chunk, the pages wholly below
    that chunk's start are dead, whatever the portions were; a long request runs in a pool of a few pages."""
    page = 8
    req = KVRequirement(1, 8, 0, chunk=chunk)
    assert req.release_window == chunk and KVRequirement(1, 8, 24, chunk=chunk).release_window == min(24, chunk)
    cm = CacheManager([CallPlan(kv=req), CallPlan(kv=KVRequirement(1, 8, 0))], max_tokens=640, page_size=page, max_requests=2,
                      device="cpu", dtype=torch.float32, max_seq_len=600, max_step_tokens=16)
    assert cm.n_groups == 2, "chunked layers have pages of their own"
    cm.admit("a")
    length = 0
    for k in [1, 2, 16, 3, 9, 16, 16, 1, 1, 7, 16, 16, 13, 2, 5, 16, 16, 16] * 2:
        cm.reserve("a", k)
        live = [p for p in cm.requests["a"].pages[0] if p >= 0]
        assert len(live) <= -(-(chunk + 16) // page) + 2
        cm.commit("a", k)
        length += k
        first = length // chunk * chunk
        for j, p in enumerate(cm.requests["a"].pages[0]):
            assert (p < 0) == ((j + 1) * page <= first), (length, j)
        assert all(p >= 0 for p in cm.requests["a"].pages[1]), "the other group keeps everything"
        cm.check_invariants()
    snap = cm.snapshot("a")
    cm.release("a")
    cm.restore("b", snap)
    assert cm.length("b") == length and cm.first_live_page("b", 0) == length // chunk * chunk // page
    cm.check_invariants()
    cm.release_all()
    assert cm.free_pages() == [80, 80]


def test_a_reader_of_a_chunked_cache_has_its_chunks():
    def build(owner, reader):
        return CacheManager([CallPlan(kv=owner), CallPlan(kv=reader, cache_from=0)], max_tokens=64, page_size=16,
                            max_requests=1, device="cpu", dtype=torch.float32)
    for reader in (KVRequirement(2, 16, 0), KVRequirement(2, 16, 8), KVRequirement(2, 16, 0, chunk=16)):
        with pytest.raises(ValueError, match="chunks"):
            build(KVRequirement(2, 16, 0, chunk=32), reader)
    build(KVRequirement(2, 16, 0, chunk=32), KVRequirement(2, 16, 0, chunk=32))
    build(KVRequirement(2, 16, 0), KVRequirement(2, 16, 0, chunk=32))
