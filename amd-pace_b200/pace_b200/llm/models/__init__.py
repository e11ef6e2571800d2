from pace_b200.llm.models import garupel, llama  # noqa: F401  (registers the architectures)
