from .engine import ServingEngine, TPServe, argmax_rows, sample_rows, sample_top_p_rows
from .hybrid import HybridEngine
from .replicas import ReplicaPlan, default_tp, make_replica_plan, split_requests


def make_engine(model, cfg=None, **kw):
    """The device-resident engine that serves ``model``: ``model.engine_class()`` where it names one, else the Llama
    engine."""
    cls = model.engine_class() if hasattr(model, "engine_class") else ServingEngine
    return cls(model, cfg, **kw)


__all__ = ["HybridEngine", "ServingEngine", "make_engine", "TPServe", "argmax_rows", "sample_rows", "sample_top_p_rows", "ReplicaPlan", "default_tp",
           "make_replica_plan", "split_requests"]
