"""Scheduler that runs exactly the portions it is told to, instead of choosing them: the replay of a
recorded schedule through the engine's own step (``LLMEngine.step``: batch assembly, model, cache and
state managers, decode graphs).  Nothing is sampled; the logits of the wanted rows ride on the step's
``SchedulerOutput``."""
from __future__ import annotations

from .request import Request, RequestStatus
from .scheduler import OmniARScheduler, ScheduledRequest, SchedulerOutput


class PortionScheduler(OmniARScheduler):
    def __init__(self, *a, **kw):
        super().__init__(*a, **kw)
        self._plan: list[tuple[Request, int, list[int]]] = []
        self.last_output: SchedulerOutput | None = None

    def plan(self, request: Request, token_ids: list[int], want=()) -> None:
        """The next step feeds ``token_ids`` as the request's next tokens; ``want``: places among them whose
        logits are asked for."""
        if not token_ids:
            raise ValueError(f"{request.request_id}: empty portion")
        if any(not 0 <= w < len(token_ids) for w in want):
            raise ValueError(f"{request.request_id}: wanted place outside the portion")
        if any(r is request for r, _, _ in self._plan):
            raise ValueError(f"{request.request_id}: two portions in one step")
        if self.max_model_len is not None and request.num_prompt_tokens + len(token_ids) > self.max_model_len:
            raise ValueError(f"{request.request_id}: longer than the model's {self.max_model_len} positions")
        request.append_prompt_chunk(token_ids)             # more chunks may follow: nothing samples
        self._plan.append((request, len(token_ids), list(want)))

    def schedule(self) -> SchedulerOutput:
        out = SchedulerOutput()
        plan, self._plan = self._plan, []
        for req, n, want in plan:
            if req in self.waiting:
                if len(self.running) >= self.max_num_seqs:
                    raise RuntimeError(f"more than {self.max_num_seqs} live requests")
                self.waiting.remove(req)
                self.running.append(req)
                req.status = RequestStatus.RUNNING
            if not self.kv.allocate_slots(req, n):
                raise RuntimeError(f"{req.request_id}: no free pages or state slots")
            start = req.num_computed_tokens
            out.scheduled.append(ScheduledRequest(req, n, start, n > 1 or start == 0, False, want))
            out.total_tokens += n
        out.finished_ids, self.finished_since_last = self.finished_since_last, []
        self.last_output = out
        return out

    def finish(self, request: Request) -> None:
        """Give back what the request holds."""
        request.status = RequestStatus.FINISHED_STOPPED
        self._release(request)
